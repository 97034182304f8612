"""Attention over one cached latent row per position with a rotated key part that all heads share."""
from __future__ import annotations

import torch

from .. import ops
from ..cache import KvRequest
from ..errors import FormatError
from ..weights.loader import ParamSpec
from .base import build_position, register_mixer, to_float32, to_run_dtype
from .projected import ProjectedMixer


class RotaryLatentMixer(ProjectedMixer):
    """q = W_q h, head by head [head_dim unrotated | rot_dim rotated]; [c | r] = W_dkv h, c RMS-normed (the latent),
    r rotated and shared by all heads. Head a: key [W_uk,a c | r], value W_uv,a c. The cache holds [c | r], one row
    a position.

    Two forms of the attention, chosen per pass:

    * over the cached rows as they are: q_a . k_a = (W_uk,a^T q_a) . c + q_a' . r, and
      sum_j p_j v_a,j = W_uv,a (sum_j p_j c_j). The queries go into the latent space head by head
      (ops.head_products), all heads attend to ONE key row whose first kv_rank elements are the values
      (ops.latent_attention), and the result leaves the latent space head by head. The cache is read once for all
      heads: decode steps, and prompts that go on from cached positions.
    * expanded, where every sequence of the pass starts at its first token and the sizes have the kernel: keys and
      values of every head are formed once (one product of the normed rows with [W_uk; W_uv]) and the queries stay as
      projected; a query and key then cost head_dim + rot_dim + value_dim products instead of 2 kv_rank + rot_dim.

    Launches: the product [q; dkv], ops.latent_write (norm, rotations, cache write), then the form's own, then
    the output product. Where the queries pass a latent of their own (spec.q_rank), the first product is [dq; dkv],
    ops.latent_write norms that latent too, and a product with W_uq and ops.latent_rotate make the query heads. Learned
    sinks (spec.sink) are an argument of the attention kernels."""
    libraries = ("elementwise", "gemm_simt", "gemm_skinny", "gemm_tc", "latent_attention", "latent_prefill_tc",
                 "attention_generic")

    def __init__(self, spec):
        s = spec
        if min(s.n_heads, s.head_dim, s.rot_dim, s.value_dim, s.kv_rank) < 1:
            raise FormatError("a latent attention with rotated keys needs positive sizes")
        if s.q_rank < 0:
            raise FormatError(f"a latent of the queries of {s.q_rank} elements")
        self.spec = spec
        self.position = build_position(spec.position)
        self.w_uk = self.w_uv = self.w_expand = self.c_gain = self.w_uq = self.q_gain = self.sinks = None

    @property
    def q_width(self):
        return self.spec.n_heads * (self.spec.head_dim + self.spec.rot_dim)

    @property
    def row(self):
        """Elements of a cached row."""
        return self.spec.kv_rank + self.spec.rot_dim

    @property
    def in_width(self):
        return ((self.spec.q_rank or self.q_width) + self.row + 7) // 8 * 8

    @property
    def out_width(self):
        return self.spec.n_heads * self.spec.value_dim

    def parameters(self):
        s, t = self.spec, self.spec.tensor
        if s.q_rank:
            out = {t["dq"]: ParamSpec((s.q_rank, s.hidden)), t["dq_norm"]: ParamSpec((s.q_rank,), "gain"),
                   t["uq"]: ParamSpec((self.q_width, s.q_rank))}
        else:
            out = {t["q"]: ParamSpec((self.q_width, s.hidden))}
        out.update({t["dkv"]: ParamSpec((self.row, s.hidden)), t["dkv_norm"]: ParamSpec((s.kv_rank,), "gain"),
                    t["uk"]: ParamSpec((s.n_heads * s.head_dim, s.kv_rank)),
                    t["uv"]: ParamSpec((s.n_heads * s.value_dim, s.kv_rank)), t["o"]: ParamSpec((s.hidden, self.out_width))})
        if s.sink:
            out[t["sink"]] = ParamSpec((s.n_heads,), "vector")
        return out

    def bind(self, tensors, dtype, device):
        s, t = self.spec, self.spec.tensor
        rows = [to_run_dtype(tensors[t[r]], dtype, device) for r in ("dq" if s.q_rank else "q", "dkv")]
        pad = self.in_width - sum(r.shape[0] for r in rows)
        if pad:
            rows.append(torch.zeros((pad, s.hidden), dtype=dtype, device=device))
        self.w_in = torch.cat(rows).contiguous()
        self.w_out = to_run_dtype(tensors[t["o"]], dtype, device)
        self.c_gain = to_float32(tensors[t["dkv_norm"]], device)
        if s.q_rank:
            self.w_uq = to_run_dtype(tensors[t["uq"]], dtype, device)
            self.q_gain = to_float32(tensors[t["dq_norm"]], device)
        if s.sink:
            self.sinks = to_float32(tensors[t["sink"]], device)
        uk = to_run_dtype(tensors[t["uk"]], dtype, device).view(s.n_heads, s.head_dim, s.kv_rank)
        uv = to_run_dtype(tensors[t["uv"]], dtype, device).view(s.n_heads, s.value_dim, s.kv_rank)
        self.w_uk = uk.transpose(1, 2).contiguous()                     # [H, kv_rank, head_dim]
        self.w_uv = uv.contiguous()                                     # [H, value_dim, kv_rank]
        self.w_expand = None
        if self._can_expand(dtype):                                     # head by head [keys; values]
            self.w_expand = torch.cat([uk, uv], dim=1).reshape(-1, s.kv_rank).contiguous()

    def prepare(self, max_positions, device):
        if self.position is not None:
            self.position.prepare(max_positions, device)

    def kv_request(self):
        return KvRequest(1, self.row, 0, values_are_keys=True)

    def mix_weights(self):
        return [w for w in (self.w_uk, self.w_uv, self.w_uq) if w is not None]

    def _shape(self, dtype, decode, fresh=False):
        s = self.spec
        return dict(decode=decode, dtype=dtype, n_heads=s.n_heads, head_dim=s.head_dim, value_dim=s.value_dim,
                    kv_rank=s.kv_rank, rot_dim=s.rot_dim, fresh=fresh)

    def _can_expand(self, dtype):
        from ..ops import tactics
        return tactics.choose_latent_attention(**self._shape(dtype, False, True)) == "latent_prefill_tc"

    def _expands(self, step, dtype) -> bool:
        """Whether a pass (a StepContext, or its host fields) runs the expanded form."""
        return (self.w_expand is not None and not step.decode and all(at == 0 for at in step.starts)
                and self._can_expand(dtype))

    def mix_replay_key(self, step):
        s, dtype = self.spec, self.w_in.dtype
        if self._expands(step, dtype):
            return ("expanded", max(step.new_counts))
        return ops.latent_attention_replay_key(step, s.n_heads)

    def mix_shapes(self, dtype, token_counts):
        s = self.spec
        heads = [(f"query product, {n} tokens", "linear",
                  dict(m=n, n=self.q_width, k=s.q_rank, in_dtype=dtype, out_dtype=dtype, lda=s.q_rank, aligned=True))
                 for n in token_counts] if s.q_rank else []
        return heads + [(label, "latent_attention", self._shape(dtype, decode, fresh))
                for label, decode, fresh in (("decode latent attention", True, False),
                                             ("prefill latent attention, first tokens", False, True),
                                             ("prefill latent attention, later tokens", False, False))]

    def mix_scratch(self, n_tokens, dtype):
        from ..engine.workspace import BufferRequest
        s = self.spec
        # phases: 0 norm, rotations, cache write; 1 queries into the latent space (or keys and values of every head);
        # 2 attention; 3 out of the latent space. Both forms of a pass share the plan.
        out = [BufferRequest("latent_q", (n_tokens, s.n_heads * self.row), dtype, 0, 2),
               BufferRequest("latent_o", (n_tokens, s.n_heads * s.kv_rank), dtype, 2, 3)]
        if self._can_expand(dtype):
            out += [BufferRequest("latent_rows", (n_tokens, self.row), dtype, 0, 2),
                    BufferRequest("latent_kv", (n_tokens, s.n_heads * (s.head_dim + s.value_dim)), dtype, 1, 2)]
        if s.q_rank:
            out += [BufferRequest("latent_cq", (n_tokens, s.q_rank), dtype, 0, 0),
                    BufferRequest("latent_heads", (n_tokens, self.q_width), dtype, 0, 2)]
        return out

    def mix(self, proj, ctx, entry, cache_entry, out, scratch):
        s = self.spec
        n, dtype = proj.shape[0], proj.dtype
        group, rows, _ = ctx.cache.layer_view(cache_entry)
        table, ring = ctx.block_tables[group], ctx.cache.table_width(group)
        angles = self.position.table if self.position is not None else None

        def buffer(name, shape):
            t = scratch(name, shape, dtype)
            return t if t is not None else torch.empty(shape, dtype=dtype, device=proj.device)

        interleaved = self.position.interleaved if self.position is not None else True
        write = dict(write_cache=(entry == cache_entry))
        common = (proj, s.n_heads, s.head_dim, s.rot_dim, s.kv_rank, self.c_gain, s.eps, angles, interleaved, ctx.tok_pos,
                  ctx.tok_seq, table, ring, rows)

        def down(queries=None, dense=None):
            """From the first product to the query heads (returned): the cached row, its dense copy, the heads' rotated
            parts (in place, or in `queries`)."""
            if not s.q_rank:
                ops.latent_write(*common, queries=queries, dense=dense, **write)
                return proj
            cq = buffer("latent_cq", (n, s.q_rank))
            ops.latent_write(*common, dense=dense, q_rank=s.q_rank, q_gain=self.q_gain, cq=cq, **write)
            up = ops.linear(cq, self.w_uq, out=buffer("latent_heads", (n, self.q_width)))
            ops.latent_rotate(up, s.n_heads, s.head_dim, s.rot_dim, s.kv_rank, angles, interleaved, ctx.tok_pos, queries=queries)
            return up

        if entry == cache_entry and self._expands(ctx, dtype):
            dense = buffer("latent_rows", (n, self.row))
            heads = down(dense=dense)                                   # the queries are rotated where they are
            kv = ops.linear(dense[:, :s.kv_rank], self.w_expand,
                            out=buffer("latent_kv", (n, s.n_heads * (s.head_dim + s.value_dim))))
            ops.latent_prefill(heads, kv, dense, s.n_heads, s.head_dim, s.rot_dim, s.value_dim, s.kv_rank, s.scale, out,
                               ctx.cu_seqlens, max(ctx.new_counts), ctx.seq_order, sinks=self.sinks)
            return
        queries = buffer("latent_q", (n, s.n_heads * self.row))
        heads = down(queries=queries)
        ops.head_products(heads, s.head_dim + s.rot_dim, self.w_uk, queries, self.row)
        latent = buffer("latent_o", (n, s.n_heads * s.kv_rank))
        ops.latent_attention(queries, rows, table, ring, ctx.tok_pos, ctx.tok_seq, s.n_heads, s.kv_rank, s.rot_dim, s.scale,
                             latent, decode=ctx.decode, seq_lens=ctx.seq_lens, max_len=ctx.max_len,
                             cu_seqlens=ctx.cu_seqlens, max_new=max(ctx.new_counts), seq_order=ctx.seq_order, sinks=self.sinks)
        ops.head_products(latent, s.kv_rank, self.w_uv, out, s.value_dim)


register_mixer("rotary_latent_attention", RotaryLatentMixer)
