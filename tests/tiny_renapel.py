"""Tiny Renapel configurations and weights for the tests.

The configurations differ in every size and option and avoid coincidences that would hide a mix-up: one to five streams and
none, value sizes on both sides of the key sizes in all three mixers, groups of 1 to 3 heads per key head, bias tables of
even and odd row counts with near and far last distances, temperatures that move within a few positions, keys and values
read by one and by two later layers, latents of the queries narrower and wider than their heads, rotated parts shorter and
longer than the unrotated ones, states with fewer and more rows than columns, one to all experts chosen from one to all of
one to four groups, limits that bite, layers without feed-forward (also the last), layer orders that start with each mixer.
"""
from __future__ import annotations

import copy
import json
import math
from pathlib import Path

import torch


def _lightning(heads, dim, vdim, decay=None):
    return {"heads": heads, "dim": dim, "vdim": vdim,
            "decay": decay if decay is not None else [1.0 - 0.5 ** (1 + 2 * h) for h in range(heads)]}


def _attention(heads, kv_heads, dim, vdim, far, temp=None, kv_from=None, scale=None):
    out = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "bias_max": far,
           "scale": scale if scale is not None else 1.0 / math.sqrt(dim)}
    if temp is not None:
        out["q_temp"] = {"coef": temp[0], "every": temp[1]}
    if kv_from is not None:
        out["kv_from"] = kv_from
    return out


def _latent(heads, dim, rot_dim, vdim, kv_rank, q_rank, base, scale=None):
    return {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank,
            "rot": {"base": base, "dims": rot_dim}, "scale": scale if scale is not None else 1.0 / math.sqrt(dim + rot_dim)}


def _moe(experts, top, ff, limit, groups=None, scale=1.0):
    router = {"experts": experts, "top": top, "scale": scale}
    if groups is not None:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "router": router, "expert": {"ff": ff, "limit": limit}}


def _layer(kind, mixer, mlp):
    return {"type": kind, "mixer": mixer, "mlp": mlp}


# P: small and odd everywhere; keys and values of layer 1 read by two later layers; two layers without feed-forward
REN_P = {
    "architecture": "Renapel", "vocab": 91, "width": 36, "norm": {"eps": 1e-4}, "streams": 2,
    "layers": [
        _layer("lightning", _lightning(3, 5, 7), _moe(6, 2, 10, 0.8, (3, 2), 1.3)),
        _layer("attention", _attention(6, 2, 6, 10, 37, (0.7, 5)), None),
        _layer("latent_attention", _latent(3, 5, 6, 7, 11, 13, 50.0), _moe(4, 1, 12, 1.5)),
        _layer("attention", _attention(2, 2, 6, 10, 20, None, 1, 0.6), _moe(5, 5, 8, 0.6, (1, 1), 0.7)),
        _layer("lightning", _lightning(2, 33, 3, [0.9, 0.35]), _moe(8, 3, 20, 2.0, (4, 2), 2.0)),
        _layer("attention", _attention(4, 2, 6, 10, 150, (0.2, 64), 1), None),
    ],
}
REN_P_ROWS = {1: 9, 3: 12, 5: 24}

# Q: sizes that tensor-core kernels take, also ones just beside them; the attention first
REN_Q = {
    "architecture": "Renapel", "vocab": 304, "width": 128, "norm": {"eps": 1e-6}, "streams": 5,
    "layers": [
        _layer("attention", _attention(4, 1, 64, 64, 90, (0.4, 33)), _moe(8, 2, 64, 1.2, (4, 1), 1.7)),
        _layer("latent_attention", _latent(4, 64, 16, 64, 80, 48, 10000.0), _moe(6, 3, 32, 0.9, (2, 2))),
        _layer("lightning", _lightning(4, 32, 48), _moe(12, 4, 64, 7.0, (3, 2), 2.5)),
        _layer("attention", _attention(6, 2, 96, 96, 300), _moe(4, 4, 32, 1.0)),
        _layer("attention", _attention(2, 1, 64, 64, 64, (0.1, 7), 0), _moe(8, 3, 96, 1.0, (2, 1), 0.5)),
        _layer("latent_attention", _latent(20, 16, 8, 24, 40, 136, 700.0, 0.11), _moe(3, 1, 64, 3.0)),
        _layer("attention", _attention(3, 1, 128, 128, 128, (1.1, 100)), None),
        _layer("lightning", _lightning(2, 72, 40, [0.999, 0.5]), _moe(16, 5, 32, 0.5, (8, 3), 1.1)),
    ],
}
REN_Q_ROWS = {0: 32, 3: 17, 4: 10, 6: 64}

# R: one layer of each kind, one stream (with weights of its own), the latent attention first
REN_R = {
    "architecture": "Renapel", "vocab": 64, "width": 32, "norm": {"eps": 1e-5}, "streams": 1,
    "layers": [
        _layer("latent_attention", _latent(1, 16, 4, 8, 8, 8, 10000.0), _moe(1, 1, 16, 1.0)),
        _layer("lightning", _lightning(1, 12, 20, [0.8]), _moe(4, 2, 24, 1.0, (2, 1))),
        _layer("attention", _attention(2, 1, 16, 24, 3, (0.5, 1)), _moe(2, 1, 8, 1.0, (2, 1), 3.0)),
    ],
}
REN_R_ROWS = {2: 4}

# S: no streams at all, three in the next
REN_S = {
    "architecture": "Renapel", "vocab": 72, "width": 64, "norm": {"eps": 1e-5},
    "layers": [
        _layer("lightning", _lightning(2, 16, 16), _moe(4, 2, 32, 1.0)),
        _layer("attention", _attention(4, 2, 32, 32, 50, (0.3, 20)), _moe(4, 2, 32, 1.0, (2, 1))),
        _layer("attention", _attention(4, 2, 32, 32, 50, None, 1), None),
    ],
}
REN_S_ROWS = {1: 16, 2: 8}

CONFIGS = {"P": (REN_P, REN_P_ROWS, 61), "Q": (REN_Q, REN_Q_ROWS, 62), "R": (REN_R, REN_R_ROWS, 63), "S": (REN_S, REN_S_ROWS, 64)}


def tensor_shapes(config, rows=None) -> dict:
    """Every tensor of a model of this configuration with its shape (written out here, not taken
    from the library). `rows`: rows of the bias table by layer (32 where it says nothing)."""
    width, streams = config["width"], config.get("streams")
    out = {"embed": (config["vocab"], width), "final.norm": (width,), "head": (config["vocab"], width)}
    for i, layer in enumerate(config["layers"]):
        m, p, q = layer["mixer"], f"l{i}.", f"l{i}.mix."

        def around(which):
            out[p + f"norm{which}"] = (width,)
            if streams is not None:
                out.update({p + f"hc{which}.in": (streams,), p + f"hc{which}.out": (streams,), p + f"hc{which}.mix": (streams, streams)})
        around(1)
        heads = m["heads"]
        if layer["type"] == "lightning":
            keys, values = heads * m["dim"], heads * m["vdim"]
            out.update({q + "q": (keys, width), q + "k": (keys, width), q + "v": (values, width), q + "g": (values, width),
                        q + "norm": (values,), q + "o": (width, values)})
        elif layer["type"] == "latent_attention":
            out.update({q + "dq": (m["q_rank"], width), q + "dq.norm": (m["q_rank"],),
                        q + "uq": (heads * (m["dim"] + m["rot_dim"]), m["q_rank"]),
                        q + "dkv": (m["kv_rank"] + m["rot_dim"], width), q + "dkv.norm": (m["kv_rank"],),
                        q + "uk": (heads * m["dim"], m["kv_rank"]), q + "uv": (heads * m["vdim"], m["kv_rank"]),
                        q + "sink": (heads,), q + "o": (width, heads * m["vdim"])})
        else:
            out.update({q + "q": (heads * m["dim"], width), q + "q.b": (heads * m["dim"],), q + "sink": (heads,),
                        q + "rel": ((rows or {}).get(i, 32), heads), q + "o": (width, heads * m["vdim"])})
            if m.get("kv_from") is None:
                keys, values = m["kv_heads"] * m["dim"], m["kv_heads"] * m["vdim"]
                out.update({q + "k": (keys, width), q + "k.b": (keys,), q + "v": (values, width), q + "v.b": (values,)})
        f = layer.get("mlp")
        if f is None:
            continue
        around(2)
        out[p + "mlp.router"] = (f["router"]["experts"], width)
        for e in range(f["router"]["experts"]):
            ff = f["expert"]["ff"]
            out.update({p + f"mlp.e{e}.gate": (ff, width), p + f"mlp.e{e}.up": (ff, width), p + f"mlp.e{e}.down": (width, ff)})
    return out


def random_weights(config, seed: int, dtype=torch.bfloat16, rows=None) -> dict:
    """Weights of a size at which every mechanism matters: projections that give values of order 1, norm weights well away
    from one, streams that stay apart, biases of the scores of order 1, sinks that hold a good part of the weight, router
    logits a few units apart."""
    gen = torch.Generator().manual_seed(seed)
    out, n = {}, config.get("streams") or 1
    for name, shape in tensor_shapes(config, rows).items():
        last = name.rsplit(".", 1)[-1]
        if last in ("norm1", "norm2", "norm"):
            t = 1.0 + 0.3 * torch.randn(shape, generator=gen)
        elif last == "in":
            t = 1.0 / n + 0.4 * torch.randn(shape, generator=gen)
        elif last == "out":
            t = 0.7 + 0.4 * torch.randn(shape, generator=gen)
        elif last == "mix":
            t = 0.8 * torch.eye(n) + 0.25 * torch.randn(shape, generator=gen)
        elif last == "rel":
            t = 1.5 * torch.randn(shape, generator=gen)
        elif last == "b":
            t = 0.5 * torch.randn(shape, generator=gen)
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
    raw, rows, seed = CONFIGS[which]
    config = copy.deepcopy(raw)
    if change is not None:
        change(config)
    weights = random_weights(config, seed, dtype, rows)
    if weights_change is not None:
        weights_change(weights)
    return write_folder(Path(tmp_path) / f"ren_{which}_{str(dtype).split('.')[-1]}", config, weights)


def random_tokens(n: int, vocab: int, seed: int) -> list:
    gen = torch.Generator().manual_seed(seed)
    return torch.randint(0, vocab, (n,), generator=gen).tolist()
