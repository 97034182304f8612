"""A plain, slow statement of the Duvozen decoder: one function per mechanism, 64-bit arithmetic, whole
sequences from their first token, its own safetensors reader. It shares no code with the package.

A layer is  x <- x + norm1(mixer(c1(x)));  x <- x + norm2(ff(c2(x))):  the norms (layer norms with a weight
and no bias) stand behind the parts only, and what a part reads is the stream plus a short causal convolution
of the stream, c(x) = x + conv(x). The mixer is a linear recurrence whose forget gate also decides what is
written, an attention over a cached latent row with a rotated key part that all heads share, or a grouped
softmax attention with head norms, a learned sink term and an element-wise gate. The feed-forward is dense
(gated, tanh-form gelu) or a routed mixture (sigmoid scores, the weight on an expert's input) with a shared
expert.
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

def layer_norm(x, weight, eps):
    """(x - mean) / sqrt(mean squared deviation + eps) * weight, over the last axis."""
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * weight


def rms_norm(x, weight, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * weight


def silu(z):
    return z / (1.0 + torch.exp(-z))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def input_conv(x, taps):
    """x [T, C] plus the causal convolution of every channel; taps [C, K], the last column at the current
    token, zeros before the sequence's start."""
    out = x.clone()
    T, K = x.shape[0], taps.shape[1]
    for j in range(K):
        back = K - 1 - j                                    # this tap reads `back` tokens ago
        if back < T:
            out[back:] += taps[:, j] * x[:T - back]
    return out


# ----------------------------------------------------------------------------- rotation

def rotary_frequencies(rot):
    """One frequency per pair, base^(-2i/dims); with a scaling, blended by bands of the pair index between the
    plain frequency and the one divided by the factor."""
    dims, base = int(rot["dims"]), float(rot["base"])
    freq = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    s = rot.get("scaling")
    if s:
        def index_of(turns):
            return dims * math.log(s["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
        lo = max(math.floor(index_of(s["fast"])), 0)
        hi = min(math.ceil(index_of(s["slow"])), dims - 1)
        for i in range(dims // 2):
            ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
            freq[i] = freq[i] / s["factor"] * ramp + freq[i] * (1.0 - ramp)
    return torch.tensor(freq, dtype=F)


def rotary_magnitude(rot):
    """What multiplies cosines and sines."""
    s = rot.get("scaling")
    return 0.1 * math.log(s["factor"]) + 1.0 if s else 1.0


def rotate(x, position, freq, interleaved, magnitude=1.0):
    """x [..., dim]: the first 2 * len(freq) elements rotate; pairs (2i, 2i + 1) or (i, i + half)."""
    half = freq.numel()
    angle = position * freq
    c, s = torch.cos(angle) * magnitude, torch.sin(angle) * magnitude
    out = x.clone()
    if interleaved:
        a, b = x[..., 0:2 * half:2], x[..., 1:2 * half:2]
        out[..., 0:2 * half:2] = a * c - b * s
        out[..., 1:2 * half:2] = b * c + a * s
    else:
        a, b = x[..., :half], x[..., half:2 * half]
        out[..., :half] = a * c - b * s
        out[..., half:2 * half] = b * c + a * s
    return out


# ----------------------------------------------------------------------------- mixers

def forget_recurrence(q, f, v, state_out=None):
    """q, f [T, H, D], v [T, H, V]: S_t = diag(f_t) S_(t-1) + (1 - f_t) v_t^T, o_t = S_t^T q_t, S zero at first."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[2], dtype=F)
    o = torch.zeros(T, H, v.shape[2], dtype=F)
    for t in range(T):
        S = f[t][:, :, None] * S + (1.0 - f[t])[:, :, None] * v[t][:, None, :]
        o[t] = (S * q[t][:, :, None]).sum(1)
    if state_out is not None:
        state_out.append(S)
    return o


def recurrence_mixer(h, m, w, p, eps, state_out=None):
    T, H, D, V = h.shape[0], int(m["heads"]), int(m["dim"]), int(m["vdim"])
    q = silu(h @ w[p + "q"].T).view(T, H, D)
    v = (h @ w[p + "v"].T).view(T, H, V)
    low = w[p + "lower"]
    f = (low + (1.0 - low) * torch.sigmoid(h @ w[p + "f"].T + w[p + "f.b"])).view(T, H, D)
    o = rms_norm(forget_recurrence(q, f, v, state_out), w[p + "norm"], eps)
    return o.reshape(T, H * V) @ w[p + "o"].T


def latent_mixer(h, m, w, p, eps):
    T, H = h.shape[0], int(m["heads"])
    D, R, V, C = int(m["dim"]), int(m["rot_dim"]), int(m["vdim"]), int(m["kv_rank"])
    q = (h @ w[p + "q"].T).view(T, H, D + R)
    down = h @ w[p + "dkv"].T
    c = rms_norm(down[:, :C], w[p + "dkv.norm"], eps)
    shared = down[:, C:].clone()                            # [T, R], one for all heads
    qr = q[:, :, D:].clone()
    rot = m.get("rot")
    if rot:
        freq, mag = rotary_frequencies(rot), rotary_magnitude(rot)
        for t in range(T):
            qr[t] = rotate(qr[t], float(t), freq, True, mag)
            shared[t] = rotate(shared[t], float(t), freq, True, mag)
    k = (c @ w[p + "uk"].T).view(T, H, D)
    v = (c @ w[p + "uv"].T).view(T, H, V)
    out = torch.zeros(T, H, V, dtype=F)
    for t in range(T):
        for a in range(H):
            scores = (k[:t + 1, a] @ q[t, a, :D] + shared[:t + 1] @ qr[t, a]) * float(m["scale"])
            out[t, a] = torch.softmax(scores, 0) @ v[:t + 1, a]
    return out.reshape(T, H * V) @ w[p + "o"].T


def sink_softmax(scores, sink):
    """Softmax with one more term in the denominator, e^sink, that has no value."""
    top = torch.maximum(scores.max(), sink)
    e = torch.exp(scores - top)
    return e / (e.sum() + torch.exp(sink - top))


def attention_mixer(h, m, w, p, eps):
    T = h.shape[0]
    H, G, D, V = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q = rms_norm((h @ w[p + "q"].T).view(T, H, D), w[p + "q.norm"], eps)
    k = rms_norm((h @ w[p + "k"].T).view(T, G, D), w[p + "k.norm"], eps)
    v = (h @ w[p + "v"].T).view(T, G, V)
    rot = m.get("rot")
    if rot:
        freq, mag = rotary_frequencies(rot), rotary_magnitude(rot)
        for t in range(T):
            q[t] = rotate(q[t], float(t), freq, False, mag)
            k[t] = rotate(k[t], float(t), freq, False, mag)
    out = torch.zeros(T, H, V, dtype=F)
    for t in range(T):
        for a in range(H):
            g = a // (H // G)
            weights = sink_softmax((k[:t + 1, g] @ q[t, a]) * float(m["scale"]), w[p + "sink"][a])
            out[t, a] = weights @ v[:t + 1, g]
    gate = torch.sigmoid(h @ w[p + "g"].T)
    return (out.reshape(T, H * V) * gate) @ w[p + "o"].T


# ----------------------------------------------------------------------------- feed-forward

def gated_ff(h, w, p, act):
    return (act(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def router(h, f, w, p):
    """Per token: the chosen experts in order of choice, their weights, and the margin of the choice."""
    top = int(f["router"]["top"])
    scores = torch.sigmoid(h @ w[p + "router"].T)
    ranked = torch.sort(scores, dim=-1, descending=True)
    margin = (ranked.values[:, top - 1] - ranked.values[:, top] if top < scores.shape[1]
              else torch.full((h.shape[0],), math.inf, dtype=F))
    return ranked.indices[:, :top], ranked.values[:, :top], margin


def routed_ff(h, f, w, p, margins=None):
    chosen, weights, margin = router(h, f, w, p)
    if margins is not None:
        margins.append(margin)
    out = gated_ff(h, w, p + "shared.", silu) if f.get("shared") else torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, s in zip(chosen[t].tolist(), weights[t]):
            out[t] += gated_ff(s * h[t], w, p + f"e{e}.", silu)          # the weight is on the input
    return out


# ----------------------------------------------------------------------------- the model

MIXERS = {"hgrn2": recurrence_mixer, "latent_attention": latent_mixer, "attention": attention_mixer}


def forward(config, w, tokens, layers_out=None, margins=None):
    """Logits [T, vocab] of one sequence from its first token; `layers_out` (a list) receives the
    stream after every layer, `margins` (a list) every routed layer's margins of choice."""
    eps = float(config["norm"]["eps"])
    scale = float(config["embedding"]["scale"]) if config.get("embedding") else 1.0
    x = w["embed"][torch.tensor(tokens, dtype=torch.long)] * scale
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}."
        y = MIXERS[layer["type"]](input_conv(x, w[p + "canon1"]), layer["mixer"], w, p + "mix.", eps)
        x = x + layer_norm(y, w[p + "norm1"], eps)
        f = layer.get("mlp")
        if f is not None:
            h = input_conv(x, w[p + "canon2"])
            y = (gated_ff(h, w, p + "mlp.", gelu_tanh) if f.get("kind", "dense") == "dense"
                 else routed_ff(h, f, w, p + "mlp.", margins))
            x = x + layer_norm(y, w[p + "norm2"], eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    return layer_norm(x, w["final.norm"], eps) @ w["head"].T * float(config.get("logit_scale", 1.0))


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
