"""Duvozen on the CPU: configuration, the plain statement's own mechanisms, and the engine's host-side logic
(packing, positions, pages, slots, the recurrence's state and the stream's last rows per layer and part, the latent
rows, the experts' rows with a shared one behind them) with the kernels replaced by their plain statements, against
the plain whole-sequence implementation."""
import copy
import math

import pytest
import torch

import plain_duvozen as plain
from tiny_duvozen import CONFIGS, DUV_P, DUV_Q, DUV_R, make_folder, random_tokens, tensor_shapes

from llm_b200.config import DuvozenConfig, config_from_dict
from llm_b200.engine import Engine, Entry, declared_parameters, load_model
from llm_b200.errors import FormatError, MissingKey, Unsupported, WeightError

TOL = dict(atol=4e-4, rtol=1e-4)


def _setup(tmp_path, which, change=None, **engine_options):
    folder = make_folder(tmp_path, which, torch.float32, change)
    config, weights = plain.read_model(folder)
    engine = Engine(load_model(folder, torch.float32, "cpu"), **{"max_tokens": 2048, **engine_options})
    return config, weights, engine


# ----------------------------------------------------------------------------- configuration

def test_config_gives_the_layers_and_names():
    config = config_from_dict(copy.deepcopy(DUV_P))
    assert isinstance(config, DuvozenConfig)
    spec = config.model_spec()
    assert [e.layer for e in spec.schedule] == list(range(6)) and spec.head == "head"
    assert spec.embedding_scale == 1.7 and spec.logit_scale == 0.6
    kinds = [b.mixer.kind for b in spec.blocks]
    assert kinds == ["forget_recurrence", "gated_attention", "rotary_latent_attention", "forget_recurrence",
                     "rotary_latent_attention", "gated_attention"]
    assert all(b.kind == "output_norm" and b.conv_taps == 4 for b in spec.blocks)
    assert spec.blocks[0].mixer_conv == "l0.canon1" and spec.blocks[0].ffn_conv == "l0.canon2"
    assert spec.blocks[0].mixer_norm.kind == "layernorm" and spec.blocks[0].mixer_norm.eps == 1e-4
    r = spec.blocks[0].mixer
    assert (r.n_heads, r.head_dim, r.value_dim, r.eps) == (3, 5, 7, 1e-4) and r.tensor["f_bias"] == "l0.mix.f.b"
    a = spec.blocks[1].mixer
    assert (a.n_heads, a.n_kv_heads, a.head_dim, a.value_dim, a.window) == (6, 2, 6, 10, 0)
    assert a.out_gate and a.sink and a.head_norm and not a.unit_sink and not a.head_gate and a.norm_eps == 1e-4
    assert a.position.pairing == "half" and a.position.rotary_dim == 4 and a.position.scaling is None
    m = spec.blocks[2].mixer
    assert (m.n_heads, m.head_dim, m.rot_dim, m.value_dim, m.kv_rank) == (3, 5, 6, 7, 11)
    assert m.position.pairing == "interleaved" and m.position.head_dim == 6
    assert dict(m.position.scaling) == {"type": "ramp", "factor": 4.0, "original": 40.0, "fast": 8.0, "slow": 1.0}
    assert m.tensor["dkv_norm"] == "l2.mix.dkv.norm" and abs(m.scale - 11 ** -0.5) < 1e-12
    routed = spec.blocks[0].feed_forward
    assert (routed.n_experts, routed.top, routed.intermediate, routed.shared.intermediate) == (5, 2, 10, 14)
    assert routed.scoring == "sigmoid" and routed.weight_on_input and routed.shared.activation == "silu"
    assert spec.blocks[4].feed_forward.shared is None
    assert spec.blocks[2].feed_forward.kind == "gated_mlp" and spec.blocks[2].feed_forward.activation == "gelu_tanh"
    assert spec.blocks[1].feed_forward is None and spec.blocks[1].ffn_norm is None and spec.blocks[1].ffn_conv is None
    nothing = config_from_dict(copy.deepcopy(DUV_R)).model_spec()
    assert nothing.embedding_scale == 1.0 and nothing.logit_scale == 1.0
    for raw in (DUV_P, DUV_Q, DUV_R):
        spec = config_from_dict(copy.deepcopy(raw)).model_spec()
        declared = {name: tuple(p.shape) for name, p in declared_parameters(spec).items()}
        assert declared == tensor_shapes(raw)
    assert config_from_dict(config.to_dict()).model_spec() == config.model_spec()


def test_config_errors_name_the_key():
    for path, value, error in [(("layers", 1, "mixer", "heads"), 5, FormatError),           # 5 heads, 2 kv heads
                               (("layers", 0, "type"), "delta", Unsupported),
                               (("layers", 0, "mlp", "kind"), "sparse", Unsupported),
                               (("layers", 1, "mixer", "rot", "dims"), 5, FormatError),
                               (("layers", 2, "mixer", "rot", "dims"), 8, FormatError),        # 6 rotated elements
                               (("layers", 0, "mlp", "router", "top"), 6, FormatError),
                               (("canon", "taps"), 0, FormatError)]:
        raw = copy.deepcopy(DUV_P)
        at = raw
        for key in path[:-1]:
            at = at[key]
        at[path[-1]] = value
        with pytest.raises(error):
            config_from_dict(raw)
    raw = copy.deepcopy(DUV_P)
    del raw["layers"][2]["mixer"]["kv_rank"]
    with pytest.raises(MissingKey) as info:
        config_from_dict(raw)
    assert "kv_rank" in str(info.value)


def test_a_missing_tensor_is_reported(tmp_path):
    def drop(weights):
        del weights["l0.mix.lower"], weights["l0.canon2"]
        weights["l0.mlp.shared.up"] = weights["l0.mlp.shared.up"][:3]
    folder = make_folder(tmp_path, "P", torch.float32, weights_change=drop)
    with pytest.raises(WeightError) as info:
        load_model(folder, torch.float32, "cpu")
    assert all(name in str(info.value) for name in ("l0.mix.lower", "l0.canon2", "l0.mlp.shared.up"))


# ----------------------------------------------------------------------------- the plain statement's mechanisms

def test_plain_mechanisms():
    gen = torch.Generator().manual_seed(0)
    F = plain.F
    x = torch.randn((7, 12), generator=gen, dtype=F) + 3.0
    y = plain.layer_norm(x, torch.ones(12, dtype=F), 1e-12)
    assert torch.allclose(y.mean(-1), torch.zeros(7, dtype=F), atol=1e-9) and torch.allclose((y * y).mean(-1), torch.ones(7, dtype=F), atol=1e-9)
    # the convolution adds to its input; the last column is the current token's tap, zeros before the start
    u = torch.randn((5, 2), generator=gen, dtype=F)
    c = plain.input_conv(u, torch.tensor([[0.0, 0.0, 1.0], [1.0, 0.0, 0.0]], dtype=F))
    assert torch.allclose(c[:, 0], 2 * u[:, 0]) and torch.allclose(c[2:, 1], u[2:, 1] + u[:3, 1]) and torch.allclose(c[:2, 1], u[:2, 1])
    # rotation: both pairings, elements beyond the rotated part stay, the magnitude multiplies what rotates
    h = torch.randn((2, 6), generator=gen, dtype=F)
    freq = plain.rotary_frequencies({"base": 50.0, "dims": 4})
    assert torch.allclose(freq, torch.tensor([1.0, 50.0 ** -0.5], dtype=F))
    for interleaved, partner in ((False, 2), (True, 1)):
        r = plain.rotate(h, 1.0, freq, interleaved, 1.5)
        assert torch.allclose(plain.rotate(h, 0.0, freq, interleaved), h) and torch.allclose(r[..., 4:], h[..., 4:])
        assert torch.allclose(r[0, 0], 1.5 * (h[0, 0] * math.cos(1.0) - h[0, partner] * math.sin(1.0)))
        assert torch.allclose(r[0, partner], 1.5 * (h[0, partner] * math.cos(1.0) + h[0, 0] * math.sin(1.0)))
    # bands: the fastest pair keeps its frequency, the slowest is slowed by the whole factor
    rot = {"base": 10000.0, "dims": 32, "scaling": {"factor": 8.0, "original": 512, "fast": 16.0, "slow": 2.0}}
    base = plain.rotary_frequencies({"base": 10000.0, "dims": 32})
    scaled = plain.rotary_frequencies(rot)
    assert torch.allclose(scaled[0], base[0]) and torch.allclose(scaled[-1], base[-1] / 8.0) and bool(((scaled <= base) & (scaled >= base / 8.0)).all())
    assert abs(plain.rotary_magnitude(rot) - (0.1 * math.log(8.0) + 1.0)) < 1e-12
    # a sink takes its share and gives nothing
    w = plain.sink_softmax(torch.zeros(3, dtype=F), torch.tensor(math.log(2.0), dtype=F))
    assert torch.allclose(w, torch.full((3,), 0.2, dtype=F))
    # the router: sigmoid scores as they are, the weight on the expert's input (not its result)
    f = {"router": {"experts": 3, "top": 2}, "shared": {"ff": 1}}
    t = {"r.router": torch.zeros((3, 2), dtype=F)}
    t["r.router"][:, 0] = torch.tensor([1.0, 3.0, 2.0], dtype=F)
    for e in ("e0", "e1", "e2", "shared"):
        t[f"r.{e}.gate"], t[f"r.{e}.up"] = torch.full((1, 2), 50.0, dtype=F), torch.full((1, 2), 2.0, dtype=F)
        t[f"r.{e}.down"] = torch.ones((2, 1), dtype=F)
    margins = []
    out = plain.routed_ff(torch.tensor([[1.0, 0.0]], dtype=F), f, t, "r.", margins)
    s = torch.sigmoid(torch.tensor([3.0, 2.0], dtype=F))
    want = 100.0 * (1.0 + (s * s).sum())                     # silu(50 s) = 50 s, times 2 s: the weight enters twice
    assert torch.allclose(out[0], want.expand(2), rtol=1e-9)
    assert abs(float(margins[0][0]) - float(s[1] - torch.sigmoid(torch.tensor(1.0, dtype=F)))) < 1e-12


def test_plain_recurrence_writes_what_it_forgets():
    F = plain.F
    q = torch.ones((3, 1, 2), dtype=F)
    f = torch.tensor([[[0.25, 1.0]], [[0.5, 0.5]], [[1.0, 0.0]]], dtype=F)
    v = torch.tensor([[[2.0]], [[4.0]], [[8.0]]], dtype=F)
    states = []
    o = plain.forget_recurrence(q, f, v, states)
    # row 0: 0.75*2 = 1.5; 0.5*1.5 + 0.5*4 = 2.75; kept. row 1: nothing written at first; 0.5*4 = 2; replaced by 8
    assert torch.allclose(states[0][0, :, 0], torch.tensor([2.75, 8.0], dtype=F))
    assert torch.allclose(o[:, 0, 0], torch.tensor([1.5, 4.75, 10.75], dtype=F))


# ----------------------------------------------------------------------------- the engine with plain kernels

@pytest.mark.parametrize("which", sorted(CONFIGS))
def test_whole_prompt_matches_plain(tmp_path, plain_kernels, which):
    config, weights, engine = _setup(tmp_path, which)
    tokens = random_tokens(140, config["vocab"], 1)
    want = plain.forward(config, weights, tokens).float()
    (slot,) = engine.acquire()
    got = engine.step([Entry(slot, tokens, list(range(len(tokens))))])
    assert torch.allclose(got, want, **TOL), float((got - want).abs().max())


@pytest.mark.parametrize("which", sorted(CONFIGS))
def test_token_by_token_equals_prefill(tmp_path, plain_kernels, which):
    config, weights, engine = _setup(tmp_path, which)
    tokens = random_tokens(75, config["vocab"], 2)
    want = plain.forward(config, weights, tokens).float()
    (slot,) = engine.acquire()
    for p, token in enumerate(tokens):                      # from the very first token on
        got = engine.step([Entry(slot, [token], [0])])
        assert torch.allclose(got[0], want[p], **TOL), (p, float((got[0] - want[p]).abs().max()))


@pytest.mark.parametrize("piece", [2, 3, 7, 64])
def test_prompts_cut_into_pieces(tmp_path, plain_kernels, piece):
    config, weights, engine = _setup(tmp_path, "P")
    tokens = random_tokens(131, config["vocab"], 3)
    want = plain.forward(config, weights, tokens).float()
    (slot,) = engine.acquire()
    for start in range(0, len(tokens), piece):
        part = tokens[start:start + piece]
        got = engine.step([Entry(slot, part, list(range(len(part))))])
        assert torch.allclose(got, want[start:start + len(part)], **TOL), start
    # the engine's own cutting of a long prompt into passes
    config, weights, engine = _setup(tmp_path, "Q", step_tokens=piece * 8)
    tokens = random_tokens(90, config["vocab"], 4)
    (slot,) = engine.acquire()
    got = engine.step([Entry(slot, tokens, [0, 50, 89])])
    assert torch.allclose(got, plain.forward(config, weights, tokens).float()[[0, 50, 89]], **TOL)


def test_unequal_batch_slot_reuse_and_early_ends(tmp_path, plain_kernels):
    config, weights, engine = _setup(tmp_path, "P", max_tokens=1024)
    lengths = [70, 1, 33, 12]
    for again in range(3):                                   # slots, pages and states are taken again
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


def test_a_mixed_step(tmp_path, plain_kernels):
    """Two sequences go on by one token while a third brings the rest of its prompt."""
    config, weights, engine = _setup(tmp_path, "Q")
    a, b, c = (random_tokens(n, config["vocab"], 40 + n) for n in (30, 9, 90))
    sa, sb, sc = engine.acquire(3)
    engine.step([Entry(sa, a[:29], []), Entry(sb, b[:8], []), Entry(sc, c[:20], [])])
    got = engine.step([Entry(sa, [a[29]], [0]), Entry(sc, c[20:], [0, 69]), Entry(sb, [b[8]], [0])])
    wa, wb, wc = (plain.forward(config, weights, s).float() for s in (a, b, c))
    want = torch.stack([wa[29], wc[20], wc[89], wb[8]])
    assert torch.allclose(got, want, **TOL), float((got - want).abs().max())


def test_a_stream_without_convolution(tmp_path, plain_kernels):
    """The arrangement's convolution is an option: a configuration without taps reads the stream as it is."""
    raw = copy.deepcopy(DUV_R)
    del raw["canon"]
    spec = config_from_dict(raw).model_spec()
    names = set(declared_parameters(spec))
    assert not any("canon" in n for n in names) and spec.blocks[0].conv_taps == 0
    from llm_b200.weights import write_random_model
    folder = write_random_model(tmp_path / "m", config_from_dict(raw), seed=3, dtype=torch.float32, std=0.3)
    config, weights = plain.read_model(folder)
    for i in range(len(raw["layers"])):                      # taps of zero: nothing is added
        for c in ("canon1", "canon2"):
            weights[f"l{i}.{c}"] = torch.zeros((raw["width"], 1), dtype=plain.F)
    engine = Engine(load_model(folder, torch.float32, "cpu"), max_tokens=256)
    tokens = random_tokens(20, raw["vocab"], 6)
    (slot,) = engine.acquire()
    got = torch.cat([engine.step([Entry(slot, tokens[:12], list(range(12)))])]
                    + [engine.step([Entry(slot, [t], [0])]) for t in tokens[12:]])
    assert torch.allclose(got, plain.forward(config, weights, tokens).float(), **TOL)


def test_random_model_writer_round_trip(tmp_path, plain_kernels):
    from llm_b200.weights import write_random_model
    config = config_from_dict(copy.deepcopy(DUV_P))
    folder = write_random_model(tmp_path / "random", config, seed=5, dtype=torch.float32, std=0.3)
    raw, weights = plain.read_model(folder)
    assert {k: tuple(v.shape) for k, v in weights.items()} == tensor_shapes(DUV_P)
    engine = Engine(load_model(folder, torch.float32, "cpu"), max_tokens=256)
    tokens = random_tokens(40, raw["vocab"], 6)
    (slot,) = engine.acquire()
    got = engine.step([Entry(slot, tokens, list(range(40)))])
    assert torch.allclose(got, plain.forward(raw, weights, tokens).float(), **TOL)


def test_inspect_and_random_commands(tmp_path, capsys):
    import json
    from llm_b200.cli import main
    (tmp_path / "config.json").write_text(json.dumps(DUV_Q))
    assert main(["random", "--config", str(tmp_path / "config.json"), "--out", str(tmp_path / "m"), "--seed", "3"]) == 0
    assert main(["inspect", str(tmp_path / "m")]) == 0
    text = capsys.readouterr().out
    assert "Duvozen" in text and "logit_scale" in text and "latent_attention" in text
