"""Tiny Duvozen configurations and weights for the tests.

The configurations differ in every size and option and avoid coincidences that would hide a mix-up: value
sizes on both sides of the key sizes in all three mixers, groups of 1, 2 and 3 heads per key head, rotated parts
shorter than a head and as long as one, plain and band-wise scaled frequencies, latents narrower and wider than
a head, recurrences whose states have fewer and more rows than columns, one to all of the experts chosen, with and
without a shared expert, layers without feed-forward (also the last), layer orders that start with each mixer,
one to five taps, embedding and logit scales that are not 1, an eps that shows.
"""
from __future__ import annotations

import copy
import json
import math
from pathlib import Path

import torch


def _attention(heads, kv_heads, dim, vdim, rot=None, scale=None):
    out = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim,
           "scale": scale if scale is not None else 1.0 / math.sqrt(dim)}
    if rot is not None:
        out["rot"] = rot
    return out


def _latent(heads, dim, rot_dim, vdim, kv_rank, base, scaling=None, scale=None):
    rot = {"base": base, "dims": rot_dim}
    if scaling is not None:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "rot": rot,
            "scale": scale if scale is not None else 1.0 / math.sqrt(dim + rot_dim)}


def _recurrence(heads, dim, vdim):
    return {"heads": heads, "dim": dim, "vdim": vdim}


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _moe(experts, top, ff, shared=None):
    out = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}
    if shared is not None:
        out["shared"] = {"ff": shared}
    return out


def _layer(kind, mixer, mlp):
    return {"type": kind, "mixer": mixer, "mlp": mlp}


# P: small and odd everywhere; the recurrence first; two layers without feed-forward, one of them the last
DUV_P = {
    "architecture": "Duvozen", "vocab": 89, "width": 36, "norm": {"eps": 1e-4}, "embedding": {"scale": 1.7},
    "logit_scale": 0.6, "canon": {"taps": 4},
    "layers": [
        _layer("hgrn2", _recurrence(3, 5, 7), _moe(5, 2, 10, 14)),
        _layer("attention", _attention(6, 2, 6, 10, {"base": 100.0, "dims": 4}), None),
        _layer("latent_attention", _latent(3, 5, 6, 7, 11, 50.0, (4.0, 40, 8.0, 1.0)), _dense(18)),
        _layer("hgrn2", _recurrence(2, 33, 3), _dense(20)),
        _layer("latent_attention", _latent(2, 9, 2, 4, 20, 3000.0), _moe(3, 3, 8)),
        _layer("attention", _attention(2, 2, 8, 4, {"base": 1000.0, "dims": 8}, 0.5), None),
    ],
}

# Q: sizes that tensor-core kernels take, also ones just beside them; the latent attention first
DUV_Q = {
    "architecture": "Duvozen", "vocab": 304, "width": 128, "norm": {"eps": 1e-6}, "embedding": {"scale": 0.8},
    "logit_scale": 1.5, "canon": {"taps": 3},
    "layers": [
        _layer("latent_attention", _latent(4, 32, 16, 48, 80, 10000.0, (6.0, 256, 16.0, 2.0)), _moe(8, 2, 64, 96)),
        _layer("attention", _attention(4, 1, 64, 64, {"base": 200000.0, "dims": 32}), _dense(160)),
        _layer("hgrn2", _recurrence(4, 32, 48), _moe(6, 1, 32, 64)),
        _layer("latent_attention", _latent(2, 64, 64, 64, 128, 500.0, scale=0.07), _dense(224)),
        _layer("attention", _attention(6, 2, 96, 96, {"base": 30000.0, "dims": 96}), _moe(4, 4, 32, 32)),
        _layer("hgrn2", _recurrence(2, 72, 40), None),
        _layer("latent_attention", _latent(20, 16, 8, 24, 40, 7000.0, (3.0, 64, 4.0, 0.5)), _dense(96)),
    ],
}

# R: one layer of each kind, no scales of its own, a single tap, attention first
DUV_R = {
    "architecture": "Duvozen", "vocab": 64, "width": 32, "norm": {"eps": 1e-5}, "canon": {"taps": 1},
    "layers": [
        _layer("attention", _attention(2, 1, 16, 24, {"base": 10.0, "dims": 2}), _dense(40)),
        _layer("latent_attention", _latent(1, 16, 4, 8, 8, 10000.0), _moe(1, 1, 16, 8)),
        _layer("hgrn2", _recurrence(1, 12, 20), _moe(4, 2, 24)),
    ],
}

CONFIGS = {"P": (DUV_P, 51), "Q": (DUV_Q, 52), "R": (DUV_R, 53)}


def tensor_shapes(config) -> dict:
    """Every tensor of a model of this configuration with its shape (written out here, not taken
    from the library)."""
    width, taps = config["width"], config["canon"]["taps"]
    out = {"embed": (config["vocab"], width), "final.norm": (width,), "head": (config["vocab"], width)}
    for i, layer in enumerate(config["layers"]):
        m, p, q = layer["mixer"], f"l{i}.", f"l{i}.mix."
        out.update({p + "norm1": (width,), p + "canon1": (width, taps)})
        heads = m["heads"]
        if layer["type"] == "hgrn2":
            keys, values = heads * m["dim"], heads * m["vdim"]
            out.update({q + "q": (keys, width), q + "f": (keys, width), q + "f.b": (keys,), q + "lower": (keys,),
                        q + "v": (values, width), q + "norm": (m["vdim"],), q + "o": (width, values)})
        elif layer["type"] == "latent_attention":
            out.update({q + "q": (heads * (m["dim"] + m["rot_dim"]), width), q + "dkv": (m["kv_rank"] + m["rot_dim"], width),
                        q + "dkv.norm": (m["kv_rank"],), q + "uk": (heads * m["dim"], m["kv_rank"]),
                        q + "uv": (heads * m["vdim"], m["kv_rank"]), q + "o": (width, heads * m["vdim"])})
        else:
            values = heads * m["vdim"]
            out.update({q + "q": (heads * m["dim"], width), q + "k": (m["kv_heads"] * m["dim"], width),
                        q + "v": (m["kv_heads"] * m["vdim"], width), q + "q.norm": (m["dim"],), q + "k.norm": (m["dim"],),
                        q + "sink": (heads,), q + "g": (values, width), q + "o": (width, values)})
        f = layer.get("mlp")
        if f is None:
            continue
        out.update({p + "norm2": (width,), p + "canon2": (width, taps)})

        def gated(prefix, ff):
            out.update({prefix + "gate": (ff, width), prefix + "up": (ff, width), prefix + "down": (width, ff)})
        if f["kind"] == "dense":
            gated(p + "mlp.", f["ff"])
            continue
        out[p + "mlp.router"] = (f["router"]["experts"], width)
        for e in range(f["router"]["experts"]):
            gated(p + f"mlp.e{e}.", f["expert"]["ff"])
        if f.get("shared"):
            gated(p + "mlp.shared.", f["shared"]["ff"])
    return out


def random_weights(config, seed: int, dtype=torch.bfloat16) -> dict:
    """Weights of a size at which every mechanism matters: projections that give values of order 1, norm weights
    well away from one, taps of order 1/2, lower bounds between none and almost one, gate biases that give short and
    long memory, sinks that hold a good part of the weight, router logits a few units apart."""
    gen = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(config).items():
        last = name.rsplit(".", 1)[-1]
        if last in ("norm1", "norm2", "norm"):
            t = 1.0 + 0.3 * torch.randn(shape, generator=gen)
        elif last in ("canon1", "canon2"):
            t = 0.6 * torch.randn(shape, generator=gen) / math.sqrt(shape[1])
        elif last == "lower":
            t = 0.9 * torch.rand(shape, generator=gen)
        elif last == "b":
            t = 1.0 + 2.0 * torch.randn(shape, generator=gen)
        elif last == "sink":
            t = 1.0 + torch.randn(shape, generator=gen)
        elif last == "router":
            t = 2.0 * torch.randn(shape, generator=gen) / math.sqrt(shape[-1])
        elif name == "embed":
            t = torch.randn(shape, generator=gen)
        else:
            t = torch.randn(shape, generator=gen) / math.sqrt(shape[-1])
        out[name] = t.to(dtype)
    return out


def write_folder(folder, config, weights) -> Path:
    from llm_b200.weights.safetensors_io import write_safetensors
    folder = Path(folder)
    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(config, indent=1))
    write_safetensors(folder / "model.safetensors", {k: v.contiguous() for k, v in weights.items()}, {"format": "pt"})
    return folder


def make_folder(tmp_path, which: str, dtype=torch.bfloat16, change=None, weights_change=None):
    """Write the folder of tiny configuration `which`; `change(config)` may alter a copy of the
    configuration first, `weights_change(weights)` the weights."""
    raw, seed = CONFIGS[which]
    config = copy.deepcopy(raw)
    if change is not None:
        change(config)
    weights = random_weights(config, seed, dtype)
    if weights_change is not None:
        weights_change(weights)
    return write_folder(Path(tmp_path) / f"duv_{which}_{str(dtype).split('.')[-1]}", config, weights)


def random_tokens(n: int, vocab: int, seed: int) -> list:
    gen = torch.Generator().manual_seed(seed)
    return torch.randint(0, vocab, (n,), generator=gen).tolist()
