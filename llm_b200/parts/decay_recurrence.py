"""Linear attention with one fixed decay per head."""
from __future__ import annotations

import torch

from .. import ops
from ..cache import StateRequest
from ..errors import FormatError
from ..weights.loader import ParamSpec
from .base import register_mixer, to_float32, to_run_dtype
from .projected import ProjectedMixer


class DecayRecurrenceMixer(ProjectedMixer):
    """Per head a state S [head_dim, value_dim], token by token
        S_t = decay S_{t-1} + k_t v_t^T,      o_t = S_t^T q_t
    with q, k and v the silu of projections; the concatenated heads are divided by their root mean square, times a weight
    per element and sigmoid(W_g h), before the output product.

    One product [q; k; v; gate] (rows padded to a multiple of 8), then ops.decay_recurrence (silu, the scan over each
    sequence's tokens, norm and gate: two launches in a decode step, three else), then the output product. Per sequence
    the cache holds S as one float32 row [heads, value_dim, head_dim]; zeroed when a slot is taken. Behind the silu
    everything is 32-bit in every run; long bfloat16 steps round q, k and v there and take the tokens of a chunk together."""
    libraries = ("elementwise", "gemm_simt", "gemm_skinny", "gemm_tc", "decay_recurrence")

    def __init__(self, spec):
        s = spec
        if min(s.n_heads, s.head_dim, s.value_dim) < 1 or len(s.decay) != s.n_heads:
            raise FormatError("a recurrence with fixed decays needs positive sizes and one decay per head")
        self.spec = spec
        self.decays = self.norm_weight = None

    @property
    def key_width(self):
        return self.spec.n_heads * self.spec.head_dim

    @property
    def out_width(self):
        return self.spec.n_heads * self.spec.value_dim

    @property
    def in_width(self):
        return (2 * self.key_width + 2 * self.out_width + 7) // 8 * 8

    def parameters(self):
        s, t, kw, vw = self.spec, self.spec.tensor, self.key_width, self.out_width
        return {t["q"]: ParamSpec((kw, s.hidden)), t["k"]: ParamSpec((kw, s.hidden)), t["v"]: ParamSpec((vw, s.hidden)),
                t["gate"]: ParamSpec((vw, s.hidden)), t["norm"]: ParamSpec((vw,), "gain"), t["o"]: ParamSpec((s.hidden, vw))}

    def bind(self, tensors, dtype, device):
        s, t = self.spec, self.spec.tensor
        rows = [to_run_dtype(tensors[t[r]], dtype, device) for r in ("q", "k", "v", "gate")]
        pad = self.in_width - sum(r.shape[0] for r in rows)
        if pad:
            rows.append(torch.zeros((pad, s.hidden), dtype=dtype, device=device))
        self.w_in = torch.cat(rows).contiguous()
        self.w_out = to_run_dtype(tensors[t["o"]], dtype, device)
        self.decays = torch.tensor(s.decay, dtype=torch.float32, device=device)
        self.norm_weight = to_float32(tensors[t["norm"]], device)

    def state_request(self):
        s = self.spec
        return StateRequest((s.n_heads * s.head_dim * s.value_dim,), torch.float32)

    def mix_weights(self):
        return [self.norm_weight]

    def mix_replay_key(self, step):
        return (bool(step.decode),)

    def mix_scratch(self, n_tokens, dtype):
        from ..engine.workspace import BufferRequest
        s = self.spec
        width = ops.decay_recurrence_work_width(s.n_heads, s.head_dim, s.value_dim)
        return [BufferRequest("decay_work", (n_tokens, width), torch.float32, 0, 0),
                BufferRequest("decay_o", (n_tokens, self.out_width), torch.float32, 0, 0)]

    def mix(self, proj, ctx, entry, cache_entry, out, scratch):
        s = self.spec
        n = proj.shape[0]
        width = ops.decay_recurrence_work_width(s.n_heads, s.head_dim, s.value_dim)
        work = scratch("decay_work", (n, width), torch.float32)
        o = scratch("decay_o", (n, self.out_width), torch.float32)
        if work is None or o is None:
            work = torch.empty((n, width), dtype=torch.float32, device=proj.device)
            o = torch.empty((n, self.out_width), dtype=torch.float32, device=proj.device)
        ops.decay_recurrence(proj, self.decays, ctx.cache.state_view(entry), ctx.cu_seqlens, ctx.slot_ids, self.norm_weight,
                             s.eps, work, o, out, s.n_heads, s.head_dim, s.value_dim, single_tokens=ctx.decode)


register_mixer("decay_recurrence", DecayRecurrenceMixer)
