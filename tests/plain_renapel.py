"""A plain, slow statement of the Renapel decoder: one function per mechanism, 64-bit arithmetic, whole
sequences from their first token, its own safetensors reader. It shares no code with the package.

A residual of several streams: a part reads a weighted sum of them, and its result is spread over their mixture.
The mixer is a linear attention with a fixed decay per head, a grouped softmax attention without rotation
(unit-size queries and keys, a temperature of the queries that grows with the position, a learned bias by distance,
a learned sink; possibly over another layer's keys and values), or an attention over a cached latent row with
queries that pass a latent of their own. The feed-forward is a mixture of clamped gated experts of which a token
chooses some, inside the best groups.
"""
from __future__ import annotations

import json
import math
import struct
from pathlib import Path

import torch

F = torch.float64


# ----------------------------------------------------------------------------- reading a folder

def read_safetensors(path) -> dict:
    data = Path(path).read_bytes()
    (n,) = struct.unpack("<Q", data[:8])
    header = json.loads(data[8:8 + n])
    out = {}
    kinds = {"BF16": torch.bfloat16, "F32": torch.float32, "I32": torch.int32, "F16": torch.float16}
    for name, info in header.items():
        if name == "__metadata__":
            continue
        a, b = info["data_offsets"]
        t = torch.frombuffer(bytearray(data[8 + n + a:8 + n + b]), dtype=kinds[info["dtype"]])
        out[name] = t.reshape(info["shape"]).to(F)
    return out


def read_model(folder):
    folder = Path(folder)
    return json.loads((folder / "config.json").read_text()), read_safetensors(folder / "model.safetensors")


# ----------------------------------------------------------------------------- small pieces

def rms_norm(x, weight, eps):
    """x over its root mean square along the last axis (eps under the root), times the weight (None: none)."""
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if weight is None else y * weight


def silu(z):
    return z / (1.0 + torch.exp(-z))


def rotate_pairs(x, position, base, dims):
    """Pairs (2i, 2i + 1) of the first `dims` elements turn by position * base^(-2i / dims)."""
    angle = torch.tensor([position * base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=F)
    c, s = torch.cos(angle), torch.sin(angle)
    out = x.clone()
    a, b = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = a * c - b * s
    out[..., 1:dims:2] = b * c + a * s
    return out


# ----------------------------------------------------------------------------- the residual streams

def read_streams(X, weights):
    """X [S, T, width]: the weighted sum over the streams."""
    return (X * weights[:, None, None]).sum(0)


def write_streams(X, y, mix, out):
    """Every stream anew from all old ones: X'_t = sum_s mix[s, t] X_s + out[t] y."""
    return torch.stack([sum(mix[s, t] * X[s] for s in range(X.shape[0])) + out[t] * y for t in range(X.shape[0])])


# ----------------------------------------------------------------------------- mixers

def decayed_attention(q, k, v, decay, state_out=None):
    """q, k [T, H, D], v [T, H, V], decay [H]: S_t = decay S_(t-1) + k_t v_t^T, o_t = S_t^T q_t, S zero at first."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[2], dtype=F)
    o = torch.zeros(T, H, v.shape[2], dtype=F)
    for t in range(T):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = (S * q[t][:, :, None]).sum(1)
    if state_out is not None:
        state_out.append(S)
    return o


def lightning_mixer(h, m, w, p, eps, kept=None, index=None, state_out=None):
    T, H, D, V = h.shape[0], int(m["heads"]), int(m["dim"]), int(m["vdim"])
    q = silu(h @ w[p + "q"].T).view(T, H, D)
    k = silu(h @ w[p + "k"].T).view(T, H, D)
    v = silu(h @ w[p + "v"].T).view(T, H, V)
    o = decayed_attention(q, k, v, torch.tensor(m["decay"], dtype=F), state_out).reshape(T, H * V)
    return (rms_norm(o, w[p + "norm"], eps) * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def bucket_of(n: int, rows: int, far: float) -> int:
    """The row of the bias table for a distance n: exact below rows / 2, then on a logarithmic scale up to `far`."""
    half = rows // 2
    if n < half:
        return n
    place = math.log(n / half) / math.log(far / half) * (rows - half)
    return min(rows - 1, half + math.floor(place + 1e-9))


def temperature(position: int, coef: float, every: float) -> float:
    return 1.0 + coef * math.log(math.floor((position + 1) / every) + 1.0)


def sink_softmax(scores, sink):
    """Softmax with one more term in the denominator, e^sink, that has no value."""
    top = torch.maximum(scores.max(), sink)
    e = torch.exp(scores - top)
    return e / (e.sum() + torch.exp(sink - top))


def attention_mixer(h, m, w, p, eps, kept=None, index=None):
    """`kept` (a dictionary): keys and values by layer index, for the layers that use another's."""
    T = h.shape[0]
    H, G, D, V = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q = rms_norm((h @ w[p + "q"].T + w[p + "q.b"]).view(T, H, D), None, eps)
    if m.get("kv_from") is not None:
        k, v = kept[int(m["kv_from"])]
    else:
        k = rms_norm((h @ w[p + "k"].T + w[p + "k.b"]).view(T, G, D), None, eps)
        v = (h @ w[p + "v"].T + w[p + "v.b"]).view(T, G, V)
        if kept is not None:
            kept[index] = (k, v)
    table, out = w[p + "rel"], torch.zeros(T, H, V, dtype=F)
    row = torch.tensor([bucket_of(n, table.shape[0], float(m["bias_max"])) for n in range(T)])
    warm = m.get("q_temp")
    for t in range(T):
        qt = q[t] * (temperature(t, float(warm["coef"]), float(warm["every"])) if warm else 1.0)
        back = row[torch.arange(t, -1, -1)]                        # the table's row for the keys 0 .. t
        for a in range(H):
            g = a // (H // G)
            scores = (k[:t + 1, g] @ qt[a]) * float(m["scale"]) + table[back, a]
            out[t, a] = sink_softmax(scores, w[p + "sink"][a]) @ v[:t + 1, g]
    return out.reshape(T, H * V) @ w[p + "o"].T


def latent_mixer(h, m, w, p, eps, kept=None, index=None):
    T, H = h.shape[0], int(m["heads"])
    D, R, V, C = int(m["dim"]), int(m["rot_dim"]), int(m["vdim"]), int(m["kv_rank"])
    q = (rms_norm(h @ w[p + "dq"].T, w[p + "dq.norm"], eps) @ w[p + "uq"].T).view(T, H, D + R)
    down = h @ w[p + "dkv"].T
    c = rms_norm(down[:, :C], w[p + "dkv.norm"], eps)
    shared, qr = down[:, C:].clone(), q[:, :, D:].clone()
    base, dims = float(m["rot"]["base"]), int(m["rot"]["dims"])
    for t in range(T):
        qr[t] = rotate_pairs(qr[t], float(t), base, dims)
        shared[t] = rotate_pairs(shared[t], float(t), base, dims)
    k = (c @ w[p + "uk"].T).view(T, H, D)
    v = (c @ w[p + "uv"].T).view(T, H, V)
    out = torch.zeros(T, H, V, dtype=F)
    for t in range(T):
        for a in range(H):
            scores = (k[:t + 1, a] @ q[t, a, :D] + shared[:t + 1] @ qr[t, a]) * float(m["scale"])
            out[t, a] = sink_softmax(scores, w[p + "sink"][a]) @ v[:t + 1, a]
    return out.reshape(T, H * V) @ w[p + "o"].T


# ----------------------------------------------------------------------------- feed-forward

def clamped_ff(h, w, p, limit):
    g = torch.clamp(h @ w[p + "gate"].T, max=limit)
    u = torch.clamp(h @ w[p + "up"].T, -limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ w[p + "down"].T


def grouped_router(h, r, weight):
    """Per token: the chosen experts in order of choice, their weights, and the margin of the choice (of the last chosen
    against the first left out, and of the last group that stays against the first that goes)."""
    n, top = int(r["experts"]), int(r["top"])
    groups = r.get("groups") or {"count": 1, "keep": 1}
    count, keep = int(groups["count"]), int(groups["keep"])
    scores = torch.softmax(h @ weight.T, dim=-1)
    T = scores.shape[0]
    best = scores.view(T, count, n // count).max(-1).values
    ranked = torch.sort(best, dim=-1, descending=True)
    allowed = torch.zeros(T, count, dtype=torch.bool)
    allowed.scatter_(1, ranked.indices[:, :keep], True)
    open_scores = torch.where(allowed[:, :, None].expand(T, count, n // count).reshape(T, n), scores, torch.tensor(-1.0, dtype=F))
    order = torch.sort(open_scores, dim=-1, descending=True)
    chosen, s = order.indices[:, :top], order.values[:, :top]
    margin = torch.full((T,), math.inf, dtype=F)
    if keep < count:
        margin = torch.minimum(margin, ranked.values[:, keep - 1] - ranked.values[:, keep])
    if top < keep * (n // count):
        margin = torch.minimum(margin, order.values[:, top - 1] - order.values[:, top])
    return chosen, s / (s.sum(-1, keepdim=True) + 1e-20) * float(r.get("scale", 1.0)), margin


def routed_ff(h, f, w, p, margins=None):
    chosen, weights, margin = grouped_router(h, f["router"], w[p + "router"])
    if margins is not None:
        margins.append(margin)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, s in zip(chosen[t].tolist(), weights[t]):
            out[t] += s * clamped_ff(h[t], w, p + f"e{e}.", float(f["expert"]["limit"]))
    return out


# ----------------------------------------------------------------------------- the model

MIXERS = {"lightning": lightning_mixer, "attention": attention_mixer, "latent_attention": latent_mixer}


def forward(config, w, tokens, layers_out=None, margins=None):
    """Logits [T, vocab] of one sequence from its first token; `layers_out` (a list) receives the
    sum of the streams after every layer, `margins` (a list) every routed layer's margins of choice."""
    eps, n_streams = float(config["norm"]["eps"]), config.get("streams")
    x = w["embed"][torch.tensor(tokens, dtype=torch.long)]
    X, kept = torch.stack([x] * int(n_streams or 1)), {}

    def sublayer(X, part, p, norm, q):
        if n_streams is None:                                       # one stream without weights of its own
            return X + part(rms_norm(X[0], w[p + norm], eps))[None]
        y = part(rms_norm(read_streams(X, w[f"{p}hc{q}.in"]), w[p + norm], eps))
        return write_streams(X, y, w[f"{p}hc{q}.mix"], w[f"{p}hc{q}.out"])

    for i, layer in enumerate(config["layers"]):
        p, f = f"l{i}.", layer.get("mlp")
        X = sublayer(X, lambda h: MIXERS[layer["type"]](h, layer["mixer"], w, p + "mix.", eps, kept, i), p, "norm1", 1)
        if f is not None:
            X = sublayer(X, lambda h: routed_ff(h, f, w, p + "mlp.", margins), p, "norm2", 2)
        if layers_out is not None:
            layers_out.append(X.sum(0))
    return rms_norm(X.sum(0), w["final.norm"], eps) @ w["head"].T


def greedy(config, w, prompt, n_new):
    """The n_new tokens that follow the prompt when the largest logit is taken every time."""
    tokens, out = list(prompt), []
    for _ in range(n_new):
        out.append(int(torch.argmax(forward(config, w, tokens)[-1])))
        tokens.append(out[-1])
    return out


def closest_call(config, w, tokens):
    """Per token, the smallest margin by which any routed layer chose its experts."""
    margins = []
    forward(config, w, tokens, margins=margins)
    if not margins:
        return torch.full((len(tokens),), math.inf, dtype=F)
    return torch.stack(margins).min(dim=0).values
