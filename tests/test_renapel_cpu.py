"""Renapel on the CPU: configuration, the plain statement's own mechanisms, and the engine's host-side logic (packing,
positions, pages, slots, the recurrence's state, keys read from another layer, the streams) with the kernels replaced by
their plain statements, against the plain whole-sequence implementation."""
import copy
import math

import pytest
import torch

import plain_ops
import plain_renapel as plain
from tiny_renapel import CONFIGS, REN_P, REN_P_ROWS, REN_Q, REN_S, make_folder, random_tokens, tensor_shapes

from llm_b200.config import RenapelConfig, config_from_dict
from llm_b200.engine import Engine, Entry, declared_parameters, load_model
from llm_b200.errors import FormatError, MissingKey, Unsupported, WeightError
from llm_b200.parts.position import distance_bucket, distance_rows, query_temperature

TOL = dict(atol=4e-4, rtol=1e-4)


def _setup(tmp_path, which, change=None, **engine_options):
    folder = make_folder(tmp_path, which, torch.float32, change)
    config, weights = plain.read_model(folder)
    engine = Engine(load_model(folder, torch.float32, "cpu"), **{"max_tokens": 2048, **engine_options})
    return config, weights, engine


# ----------------------------------------------------------------------------- configuration

def test_config_gives_the_layers_and_names():
    config = config_from_dict(copy.deepcopy(REN_P))
    assert isinstance(config, RenapelConfig)
    spec = config.model_spec()
    assert spec.streams == 2 and spec.head == "head" and all(b.kind == "streams" and b.n_streams == 2 for b in spec.blocks)
    assert [(e.layer, e.cache_of) for e in spec.schedule] == [(0, None), (1, None), (2, None), (3, 1), (4, None), (5, 1)]
    assert [b.mixer.kind for b in spec.blocks] == ["decay_recurrence", "gated_attention", "rotary_latent_attention",
                                                   "gated_attention", "decay_recurrence", "gated_attention"]
    r = spec.blocks[4].mixer
    assert (r.n_heads, r.head_dim, r.value_dim, r.decay, r.eps) == (2, 33, 3, (0.9, 0.35), 1e-4)
    a = spec.blocks[1].mixer
    assert (a.n_heads, a.n_kv_heads, a.head_dim, a.value_dim, a.window) == (6, 2, 6, 10, 0)
    assert a.bias and a.unit_norm and a.sink and not (a.head_norm or a.out_gate or a.shared_kv) and a.position is None
    assert a.q_temp == (0.7, 5.0) and a.distance_bias == 37.0 and a.tensor["k_bias"] == "l1.mix.k.b"
    assert spec.blocks[3].mixer.shared_kv and spec.blocks[3].mixer.q_temp is None and spec.blocks[3].mixer.scale == 0.6
    m = spec.blocks[2].mixer
    assert (m.n_heads, m.head_dim, m.rot_dim, m.value_dim, m.kv_rank, m.q_rank, m.sink) == (3, 5, 6, 7, 11, 13, True)
    assert m.position.pairing == "interleaved" and m.position.theta == 50.0 and m.tensor["uq"] == "l2.mix.uq"
    f = spec.blocks[0].feed_forward
    assert (f.n_experts, f.top, f.groups, f.keep_groups, f.out_scale, f.intermediate) == (6, 2, 3, 2, 1.3, 10)
    assert f.scoring == "all" and f.activation == "clamped" and f.limit == 0.8 and f.alpha == 1.702 and not f.correction
    assert spec.blocks[2].feed_forward.groups == 1 and spec.blocks[2].feed_forward.keep_groups == 1
    assert spec.blocks[1].feed_forward is None and spec.blocks[1].ffn_streams is None and spec.blocks[1].ffn_norm is None
    assert dict(spec.blocks[0].ffn_streams) == {"in": "l0.hc2.in", "mix": "l0.hc2.mix", "out": "l0.hc2.out"}
    plain_residual = config_from_dict(copy.deepcopy(REN_S)).model_spec()
    assert plain_residual.streams == 0 and all(b.kind == "pre_norm" for b in plain_residual.blocks)
    for raw, rows, _ in CONFIGS.values():
        spec = config_from_dict(copy.deepcopy(raw)).model_spec()
        declared = declared_parameters(spec)
        shapes = tensor_shapes(raw, rows)
        assert declared.keys() == shapes.keys() and all(p.fits(shapes[name]) for name, p in declared.items())
        assert tensor_shapes(raw) == {name: tuple(p.shape) for name, p in declared.items()}
    assert config_from_dict(config.to_dict()).model_spec() == config.model_spec()


def test_config_errors_name_the_key():
    for path, value, error in [(("layers", 1, "mixer", "heads"), 5, FormatError),           # 5 heads, 2 kv heads
                               (("layers", 0, "type"), "delta", Unsupported),
                               (("layers", 0, "mlp", "kind"), "dense", Unsupported),
                               (("layers", 0, "mixer", "decay"), [0.5], FormatError),          # 3 heads
                               (("layers", 2, "mixer", "rot", "dims"), 8, FormatError),        # 6 rotated elements
                               (("layers", 0, "mlp", "router", "top"), 5, FormatError),        # 2 groups of 2 stay
                               (("layers", 0, "mlp", "router", "groups", "count"), 4, FormatError),
                               (("layers", 0, "mlp", "router", "groups", "keep"), 4, FormatError),
                               (("layers", 3, "mixer", "kv_from"), 3, FormatError),            # itself
                               (("layers", 3, "mixer", "kv_from"), 0, FormatError),            # no attention
                               (("layers", 5, "mixer", "kv_from"), 3, FormatError),            # no keys of its own
                               (("layers", 3, "mixer", "vdim"), 6, FormatError),               # read from values of 10
                               (("streams",), 0, FormatError)]:
        raw = copy.deepcopy(REN_P)
        at = raw
        for key in path[:-1]:
            at = at[key]
        at[path[-1]] = value
        with pytest.raises(error):
            config_from_dict(raw)
    raw = copy.deepcopy(REN_P)
    del raw["layers"][2]["mixer"]["q_rank"]
    with pytest.raises(MissingKey) as info:
        config_from_dict(raw)
    assert "q_rank" in str(info.value)


def test_tensors_that_do_not_fit_are_reported(tmp_path):
    def spoil(weights):
        del weights["l0.hc1.mix"], weights["l2.mix.dq.norm"]
        weights["l1.mix.rel"] = weights["l1.mix.rel"][:, :3]            # its rows are free, its heads are not
        weights["l3.mix.k"] = torch.zeros((12, 36))                      # a layer that reads another's keys has none
    folder = make_folder(tmp_path, "P", torch.float32, weights_change=spoil)
    with pytest.raises(WeightError) as info:
        load_model(folder, torch.float32, "cpu")
    assert all(name in str(info.value) for name in ("l0.hc1.mix", "l2.mix.dq.norm", "l1.mix.rel", "l3.mix.k"))

    def many(weights):
        weights["l1.mix.rel"] = torch.zeros((80, 6))                     # half of the rows reach beyond the farthest distance
    folder = make_folder(tmp_path / "b", "P", torch.float32, weights_change=many)
    with pytest.raises(FormatError):
        load_model(folder, torch.float32, "cpu")


# ----------------------------------------------------------------------------- mechanisms

def test_distance_buckets():
    """Exact below half of the rows, the last row from the farthest distance on, every distance between on the logarithmic
    scale; edges that lie on a whole step belong to the bucket that starts there."""
    assert [distance_bucket(n, 8, 64.0) for n in (0, 1, 3, 4, 7, 8, 15, 16, 31, 32, 63, 64, 1000)] == [0, 1, 3, 4, 4, 5, 5, 6, 6, 7, 7, 7, 7]
    for rows, far in ((32, 120.0), (9, 37.0), (24, 150.0), (17, 300.0), (2, 5.0), (64, 128.0), (16, 1 << 14)):
        table = distance_rows(rows, far)
        assert table[-1] == rows - 1 and table.count(rows - 1) == 1 and len(table) <= far + 1
        assert table == sorted(table) and table[:rows // 2] == list(range(rows // 2))
        for n, bucket in enumerate(table):
            assert bucket == plain.bucket_of(n, rows, far)
        assert plain.bucket_of(len(table) + 5, rows, far) == rows - 1
    assert distance_rows(1, 5.0) == [0]


def test_query_temperatures():
    t = query_temperature(40, 0.5, 8.0)
    want = [plain.temperature(p, 0.5, 8.0) for p in range(40)]
    assert torch.allclose(t, torch.tensor(want)) and float(t[6]) == 1.0 and float(t[7]) > 1.3 and float(t[15]) > float(t[14])


def test_plain_mechanisms():
    gen = torch.Generator().manual_seed(0)
    F = plain.F
    # streams: the mixture goes from the first index to the second; the result is spread over all
    X = torch.randn((2, 1, 3), generator=gen, dtype=F)
    mix, out = torch.tensor([[1.0, 2.0], [0.0, 3.0]], dtype=F), torch.tensor([0.5, -1.0], dtype=F)
    y = torch.randn((1, 3), generator=gen, dtype=F)
    N = plain.write_streams(X, y, mix, out)
    assert torch.allclose(N[0], X[0] + 0.5 * y) and torch.allclose(N[1], 2 * X[0] + 3 * X[1] - y)
    assert torch.allclose(plain.read_streams(X, torch.tensor([2.0, -1.0], dtype=F)), 2 * X[0] - X[1])
    # the recurrence: fades by the head's decay, then writes
    states = []
    o = plain.decayed_attention(torch.ones((2, 1, 1), dtype=F), torch.tensor([[[2.0]], [[3.0]]], dtype=F),
                                torch.tensor([[[5.0]], [[7.0]]], dtype=F), torch.tensor([0.5], dtype=F), states)
    assert o[:, 0, 0].tolist() == [10.0, 26.0] and float(states[0]) == 26.0
    # rotation of neighbouring pairs
    h = torch.randn((2, 6), generator=gen, dtype=F)
    r = plain.rotate_pairs(h, 3.0, 50.0, 4)
    assert torch.allclose(r[:, 4:], h[:, 4:]) and torch.allclose(plain.rotate_pairs(h, 0.0, 50.0, 4), h)
    angle = 3.0 * 50.0 ** -0.5
    assert torch.allclose(r[:, 2], h[:, 2] * math.cos(angle) - h[:, 3] * math.sin(angle))
    assert torch.allclose(r[:, 3], h[:, 3] * math.cos(angle) + h[:, 2] * math.sin(angle))
    # a sink takes its share and gives nothing
    w = plain.sink_softmax(torch.zeros(3, dtype=F), torch.tensor(math.log(2.0), dtype=F))
    assert torch.allclose(w, torch.full((3,), 0.2, dtype=F))
    # clamped experts: the gate has an upper bound alone, the other factor both
    p = {"e.gate": torch.eye(3, dtype=F), "e.up": torch.eye(3, dtype=F), "e.down": torch.eye(3, dtype=F)}
    got = plain.clamped_ff(torch.tensor([[5.0, -5.0, 0.5]], dtype=F), p, "e.", 1.0)[0]
    sig = lambda z: 1.0 / (1.0 + math.exp(-z))
    assert torch.allclose(got, torch.tensor([sig(1.702) * 2.0, 0.0, 0.5 * sig(0.851) * 1.5], dtype=F))
    assert abs(plain.clamped_ff(torch.tensor([[-5.0, 0.0, 0.0]], dtype=F), {**p, "e.up": -p["e.up"]}, "e.", 1.0)[0, 0]
               - (-5.0 * sig(-8.51) * 2.0)) < 1e-12
    # groups: the best single score decides which group stays, not the sum
    weight = torch.log(torch.tensor([[0.30], [0.01], [0.20], [0.19], [0.02], [0.28]], dtype=F))
    chosen, shares, margin = plain.grouped_router(torch.ones((1, 1), dtype=F), {"experts": 6, "top": 2, "scale": 3.0,
                                                                                "groups": {"count": 3, "keep": 2}}, weight)
    assert chosen.tolist() == [[0, 5]] and torch.allclose(shares, torch.tensor([[3 * 0.30 / 0.58, 3 * 0.28 / 0.58]], dtype=F))
    assert abs(float(margin[0]) - 0.08) < 1e-12
    chosen, _, _ = plain.grouped_router(torch.ones((1, 1), dtype=F), {"experts": 6, "top": 2, "groups": {"count": 3, "keep": 1}}, weight)
    assert chosen.tolist() == [[0, 1]]


def test_the_kernels_plain_statement_of_the_router_agrees():
    """tests/plain_ops (what the GPU kernels are compared with) beside the plain model's router, groups included."""
    gen = torch.Generator().manual_seed(3)
    for experts, top, count, keep in ((12, 3, 3, 2), (8, 4, 4, 3), (6, 6, 1, 1), (9, 2, 9, 4), (16, 1, 2, 1)):
        h, router = torch.randn((20, 10), generator=gen), torch.randn((experts, 10), generator=gen)
        a = 20 * top
        ids, weights = torch.zeros(a, dtype=torch.int32), torch.zeros(a)
        plain_ops.routed_experts(h, router, None, torch.zeros((experts, 4, 10)), torch.zeros((experts, 10, 2)), top, ids, weights, None,
                                 None, None, torch.zeros((a, 10)), scoring=1, weight_scale=1.4, groups=count, keep=keep, limit=1.0)
        chosen, shares, _ = plain.grouped_router(h.double(), {"experts": experts, "top": top, "scale": 1.4,
                                                              "groups": {"count": count, "keep": keep}}, router.double())
        assert torch.equal(ids.view(20, top).long(), chosen) and torch.allclose(weights.view(20, top).double(), shares, atol=1e-6)


# ----------------------------------------------------------------------------- the engine with plain kernels

@pytest.mark.parametrize("which", sorted(CONFIGS))
def test_whole_prompt_matches_plain(tmp_path, plain_kernels, which):
    config, weights, engine = _setup(tmp_path, which)
    tokens = random_tokens(110, config["vocab"], 1)
    want = plain.forward(config, weights, tokens).float()
    (slot,) = engine.acquire()
    got = engine.step([Entry(slot, tokens, list(range(len(tokens))))])
    assert torch.allclose(got, want, **TOL), float((got - want).abs().max())


@pytest.mark.parametrize("which", sorted(CONFIGS))
def test_token_by_token_equals_prefill(tmp_path, plain_kernels, which):
    config, weights, engine = _setup(tmp_path, which)
    tokens = random_tokens(70, config["vocab"], 2)
    want = plain.forward(config, weights, tokens).float()
    (slot,) = engine.acquire()
    for p, token in enumerate(tokens):                      # from the very first token on
        got = engine.step([Entry(slot, [token], [0])])
        assert torch.allclose(got[0], want[p], **TOL), (p, float((got[0] - want[p]).abs().max()))


@pytest.mark.parametrize("piece", [2, 7, 64])
def test_prompts_cut_into_pieces(tmp_path, plain_kernels, piece):
    config, weights, engine = _setup(tmp_path, "P")
    tokens = random_tokens(100, config["vocab"], 3)
    want = plain.forward(config, weights, tokens).float()
    (slot,) = engine.acquire()
    for start in range(0, len(tokens), piece):
        part = tokens[start:start + piece]
        got = engine.step([Entry(slot, part, list(range(len(part))))])
        assert torch.allclose(got, want[start:start + len(part)], **TOL), start
    # the engine's own cutting of a long prompt into passes
    config, weights, engine = _setup(tmp_path, "R", step_tokens=piece * 4)
    tokens = random_tokens(90, config["vocab"], 4)
    (slot,) = engine.acquire()
    got = engine.step([Entry(slot, tokens, [0, 50, 89])])
    assert torch.allclose(got, plain.forward(config, weights, tokens).float()[[0, 50, 89]], **TOL)


def test_unequal_batch_slot_reuse_and_early_ends(tmp_path, plain_kernels):
    config, weights, engine = _setup(tmp_path, "P", max_tokens=1024)
    lengths = [70, 1, 33, 12]
    for again in range(2):                                   # slots, pages and states are taken again
        seqs = [random_tokens(n, config["vocab"], 10 * again + n) for n in lengths]
        want = [plain.forward(config, weights, s).float() for s in seqs]
        slots = engine.acquire(len(seqs))
        heads = [max(1, n - 5 - i) for i, n in enumerate(lengths)]
        got = engine.step([Entry(s, q[:h], [h - 1]) for s, q, h in zip(slots, seqs, heads)])
        for b, h in enumerate(heads):
            assert torch.allclose(got[b], want[b][h - 1], **TOL), (again, b)
        live = [b for b in range(len(seqs)) if heads[b] < lengths[b]]
        engine.release([slots[b] for b in range(len(seqs)) if b not in live])
        done = 0
        while live:
            got = engine.step([Entry(slots[b], [seqs[b][heads[b] + done]], [0]) for b in live])
            for r, b in enumerate(live):
                assert torch.allclose(got[r], want[b][heads[b] + done], **TOL), (again, b, done)
            done += 1
            ended = [b for b in live if heads[b] + done == lengths[b]]
            engine.release([slots[b] for b in ended])
            live = [b for b in live if b not in ended]
        engine.cache.check()
        assert engine.cache.slots.n_held == 0


def test_layers_that_read_other_layers_keys_hold_no_cache(tmp_path, plain_kernels):
    config, weights, engine = _setup(tmp_path, "P")
    assert engine.cache.entry_group[1] is not None and engine.cache.entry_group[3] is None and engine.cache.entry_group[5] is None
    assert engine.model.blocks[3].mixer.w_in.shape[0] == 16                     # 2 heads of 6 in rows of 8


def test_random_model_writer_round_trip(tmp_path, plain_kernels):
    from llm_b200.weights import write_random_model
    for raw in (REN_P, REN_S):
        folder = write_random_model(tmp_path / f"random{raw['vocab']}", config_from_dict(
            {**copy.deepcopy(raw), "layers": copy.deepcopy(raw["layers"][:4])}), seed=5, dtype=torch.float32, std=0.3, gain_noise=0.2)
        config, weights = plain.read_model(folder)
        engine = Engine(load_model(folder, torch.float32, "cpu"), max_tokens=256)
        tokens = random_tokens(40, raw["vocab"], 6)
        (slot,) = engine.acquire()
        got = engine.step([Entry(slot, tokens, list(range(40)))])
        assert torch.allclose(got, plain.forward(config, weights, tokens).float(), **TOL)


def test_streams_need_a_model_of_streams():
    from dataclasses import replace
    from llm_b200.engine.model import DecoderModel
    spec = config_from_dict(copy.deepcopy(REN_P)).model_spec()
    for wrong in (replace(spec, streams=3), replace(spec, streams=0),
                  replace(spec, schedule=(spec.schedule[0], replace(spec.schedule[1], add_embedding=True)) + spec.schedule[2:])):
        with pytest.raises(FormatError):
            DecoderModel(wrong)
    with pytest.raises(Unsupported):
        DecoderModel(config_from_dict({**copy.deepcopy(REN_P), "streams": 17}).model_spec())


def test_inspect_and_random_commands(tmp_path, capsys):
    import json
    from llm_b200.cli import main
    (tmp_path / "config.json").write_text(json.dumps(REN_Q))
    assert main(["random", "--config", str(tmp_path / "config.json"), "--out", str(tmp_path / "m"), "--seed", "3"]) == 0
    assert main(["inspect", str(tmp_path / "m")]) == 0
    text = capsys.readouterr().out
    assert "Renapel" in text and "latent_attention" in text
