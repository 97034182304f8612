"""Linear attention whose forget gate also decides what is written."""
from __future__ import annotations

import torch

from .. import ops
from ..cache import StateRequest
from ..errors import FormatError
from ..weights.loader import ParamSpec
from .base import register_mixer, to_float32, to_run_dtype
from .projected import ProjectedMixer


class ForgetRecurrenceMixer(ProjectedMixer):
    """Per head a state S [head_dim, value_dim], token by token
        S_t = diag(f_t) S_{t-1} + (1 - f_t) v_t^T,      o_t = S_t^T q_t
    with q = silu(W_q h), v = W_v h and f = l + (1 - l) sigmoid(W_f h + b), l a stored lower bound per head and
    channel; every head's o is divided by its root mean square, times a weight that the heads share, before the
    output product (Qin et al., "HGRN2: Gated Linear RNNs with State Expansion").

    One product [q; f; v] (rows padded to a multiple of 8), then ops.forget_recurrence (the gates, the scan over each
    sequence's tokens, the heads' norm: one launch in a decode step, three else), then the output product. Per
    sequence the cache holds S as one float32 row [heads, value_dim, head_dim]; zeroed when a slot is taken.
    Everything behind the projection is 32-bit in every run."""
    libraries = ("elementwise", "gemm_simt", "gemm_skinny", "gemm_tc", "forget_recurrence")

    def __init__(self, spec):
        s = spec
        if min(s.n_heads, s.head_dim, s.value_dim) < 1:
            raise FormatError("a forget-gated recurrence needs positive sizes")
        self.spec = spec
        self.f_bias = self.lower = self.norm_weight = None

    @property
    def key_width(self):
        return self.spec.n_heads * self.spec.head_dim

    @property
    def out_width(self):
        return self.spec.n_heads * self.spec.value_dim

    @property
    def in_width(self):
        return (2 * self.key_width + self.out_width + 7) // 8 * 8

    def parameters(self):
        s, t, kw, vw = self.spec, self.spec.tensor, self.key_width, self.out_width
        return {t["q"]: ParamSpec((kw, s.hidden)), t["f"]: ParamSpec((kw, s.hidden)), t["f_bias"]: ParamSpec((kw,), "bias"),
                t["lower"]: ParamSpec((kw,), "vector"), t["v"]: ParamSpec((vw, s.hidden)),
                t["norm"]: ParamSpec((s.value_dim,), "gain"), t["o"]: ParamSpec((s.hidden, vw))}

    def bind(self, tensors, dtype, device):
        s, t = self.spec, self.spec.tensor
        rows = [to_run_dtype(tensors[t[r]], dtype, device) for r in ("q", "f", "v")]
        pad = self.in_width - sum(r.shape[0] for r in rows)
        if pad:
            rows.append(torch.zeros((pad, s.hidden), dtype=dtype, device=device))
        self.w_in = torch.cat(rows).contiguous()
        self.w_out = to_run_dtype(tensors[t["o"]], dtype, device)
        self.f_bias = to_float32(tensors[t["f_bias"]], device)
        self.lower = to_float32(tensors[t["lower"]], device)
        self.norm_weight = to_float32(tensors[t["norm"]], device)

    def state_request(self):
        s = self.spec
        return StateRequest((s.n_heads * s.head_dim * s.value_dim,), torch.float32)

    def mix_replay_key(self, step):
        return (bool(step.decode),)

    def mix_scratch(self, n_tokens, dtype):
        from ..engine.workspace import BufferRequest
        s = self.spec
        width = ops.forget_recurrence_work_width(s.n_heads, s.head_dim, s.value_dim)
        return [BufferRequest("forget_work", (n_tokens, width), torch.float32, 0, 0),
                BufferRequest("forget_o", (n_tokens, self.out_width), torch.float32, 0, 0)]

    def mix(self, proj, ctx, entry, cache_entry, out, scratch):
        s = self.spec
        n = proj.shape[0]
        width = ops.forget_recurrence_work_width(s.n_heads, s.head_dim, s.value_dim)
        work = scratch("forget_work", (n, width), torch.float32)
        o = scratch("forget_o", (n, self.out_width), torch.float32)
        if work is None or o is None:
            work = torch.empty((n, width), dtype=torch.float32, device=proj.device)
            o = torch.empty((n, self.out_width), dtype=torch.float32, device=proj.device)
        ops.forget_recurrence(proj, self.f_bias, self.lower, ctx.cache.state_view(entry), ctx.cu_seqlens, ctx.slot_ids,
                              self.norm_weight, s.eps, work, o, out, s.n_heads, s.head_dim, s.value_dim,
                              single_tokens=ctx.decode)


register_mixer("forget_recurrence", ForgetRecurrenceMixer)
