"""Configuration of the Renapel decoder, read from its own config.json keys.

A Renapel model has a residual of several streams (`streams`): every part reads a weighted sum of them behind an RMS norm,
and its result is spread over a mixture of them (without the key: one stream, x += part(norm(x))). A layer's `type`
names its mixer: `lightning` (linear attention with one fixed decay per head and an element-wise gate), `attention` (grouped
softmax attention without rotation: unit-size queries and keys, a temperature of the queries by position, a learned bias by
distance, a learned sink; `kv_from` names the layer whose keys and values it reads) or `latent_attention` (attention over
one cached latent row with a rotated key part that all heads share, queries through a latent of their own, a learned sink).
Its `mlp` is `moe` (clamped gated experts, softmax scores over all of them, chosen inside the best groups of neighbours) or
null. The head is a matrix of its own.
"""
from __future__ import annotations

import json
from dataclasses import dataclass
from typing import Optional

from ..errors import FormatError, Unsupported
from ..parts.spec import (BlockSpec, DecayRecurrenceSpec, GatedAttentionSpec, ModelSpec, NormSpec, PositionSpec,
                          RotaryLatentSpec, RoutedExpertsSpec, ScheduleEntry, StreamsBlockSpec, names)
from .base import ConfigReader

# no key of the configuration bounds a sequence: the engine's context does
MAX_POSITIONS = 1 << 22
# the slope of the experts' sigmoid
GATE_SLOPE = 1.702


@dataclass(frozen=True)
class RenapelConfig:
    """`layers` keeps the configuration's list as JSON text per layer (hashable); the typed view is `model_spec()`."""
    vocab: int
    width: int
    eps: float
    streams: Optional[int]
    layers: tuple

    architecture = "Renapel"

    @classmethod
    def from_dict(cls, raw: dict, where: str = "config.json") -> "RenapelConfig":
        r = ConfigReader(raw, where)
        layers = raw.get("layers")
        if not isinstance(layers, list) or not layers:
            raise FormatError(f"{where}: 'layers' must be a non-empty list")
        norm = ConfigReader(r.mapping("norm"), f"{where}: norm")
        config = cls(vocab=r.integer("vocab", minimum=1), width=r.integer("width", minimum=1),
                     eps=norm.number("eps", positive=True),
                     streams=r.integer("streams", minimum=1) if raw.get("streams") is not None else None,
                     layers=tuple(json.dumps(layer, sort_keys=True) for layer in layers))
        config.model_spec()            # every layer is read once here, so that a bad key is reported at load
        return config

    def to_dict(self) -> dict:
        out = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps},
               "layers": [json.loads(text) for text in self.layers]}
        if self.streams is not None:
            out["streams"] = self.streams
        return out

    def to_json(self) -> str:
        return json.dumps(self.to_dict(), indent=2) + "\n"

    # ------------------------------------------------------------------ the model as data

    def _recurrence(self, p: str, raw: dict, where: str):
        m = ConfigReader(raw, where)
        heads, decay = m.integer("heads", minimum=1), raw.get("decay")
        if not isinstance(decay, list) or len(decay) != heads or any(
                isinstance(d, bool) or not isinstance(d, (int, float)) for d in decay):
            raise FormatError(f"{where}: 'decay' must be a list of {heads} numbers, one per head")
        return DecayRecurrenceSpec(
            hidden=self.width, n_heads=heads, head_dim=m.integer("dim", minimum=1), value_dim=m.integer("vdim", minimum=1),
            decay=tuple(float(d) for d in decay), eps=self.eps,
            names=names(q=p + "q", k=p + "k", v=p + "v", gate=p + "g", norm=p + "norm", o=p + "o"))

    def _attention(self, p: str, raw: dict, where: str, source: Optional[dict]):
        """`source`: the mixer of the layer whose keys and values this one reads (None: its own)."""
        m = ConfigReader(raw, where)
        heads, kv_heads = m.integer("heads", minimum=1), m.integer("kv_heads", minimum=1)
        if heads % kv_heads:
            raise FormatError(f"{where}: {heads} heads are no multiple of {kv_heads} kv_heads")
        dim = m.integer("dim", minimum=1)
        vdim = m.integer("vdim", dim, minimum=1)
        if source is not None:
            s = ConfigReader(source, where)
            if (s.integer("kv_heads"), s.integer("dim"), s.integer("vdim", s.integer("dim"))) != (kv_heads, dim, vdim):
                raise FormatError(f"{where}: keys and values read from a layer of other sizes")
        temp, raw_temp = None, m.mapping("q_temp", None)
        if raw_temp is not None:
            t = ConfigReader(raw_temp, f"{where}: q_temp")
            temp = (t.number("coef"), t.number("every", positive=True))
        return GatedAttentionSpec(
            hidden=self.width, n_heads=heads, n_kv_heads=kv_heads, head_dim=dim, value_dim=vdim, scale=m.number("scale", positive=True),
            window=0, values_are_keys=False, out_gate=False, position=None, norm_eps=self.eps, unit_norm=True, bias=True,
            q_temp=temp, sink=True, shared_kv=source is not None,
            distance_bias=m.number("bias_max", positive=True),
            names=names(q=p + "q", k=p + "k", v=p + "v", o=p + "o", q_bias=p + "q.b", k_bias=p + "k.b", v_bias=p + "v.b",
                        rel=p + "rel", sink=p + "sink"))

    def _latent(self, p: str, raw: dict, where: str):
        m = ConfigReader(raw, where)
        rot_dim = m.integer("rot_dim", minimum=1)
        rot = ConfigReader(m.mapping("rot"), f"{where}: rot")
        dims = rot.integer("dims", rot_dim, minimum=2)
        if dims % 2 or dims > rot_dim:
            raise FormatError(f"{where}: rot.dims {dims} must be even and at most {rot_dim}")
        return RotaryLatentSpec(
            hidden=self.width, n_heads=m.integer("heads", minimum=1), head_dim=m.integer("dim", minimum=1),
            rot_dim=rot_dim, value_dim=m.integer("vdim", minimum=1), kv_rank=m.integer("kv_rank", minimum=1),
            q_rank=m.integer("q_rank", minimum=1), scale=m.number("scale", positive=True), eps=self.eps, sink=True,
            position=PositionSpec(head_dim=rot_dim, theta=rot.number("base", positive=True), max_positions=MAX_POSITIONS,
                                  pairing="interleaved", rotary_dim=dims),
            names=names(dq=p + "dq", dq_norm=p + "dq.norm", uq=p + "uq", dkv=p + "dkv", dkv_norm=p + "dkv.norm",
                        uk=p + "uk", uv=p + "uv", sink=p + "sink", o=p + "o"))

    def _feed_forward(self, p: str, raw: dict, where: str):
        f = ConfigReader(raw, where)
        kind = f.string("kind", "moe")
        if kind != "moe":
            raise Unsupported(f"{where}: kind '{kind}' (built: 'moe')")
        router = ConfigReader(f.mapping("router"), f"{where}: router")
        expert = ConfigReader(f.mapping("expert"), f"{where}: expert")
        groups = router.mapping("groups", None)
        g = ConfigReader(groups if groups is not None else {"count": 1, "keep": 1}, f"{where}: router.groups")
        experts, top = router.integer("experts", minimum=1), router.integer("top", minimum=1)
        count, keep = g.integer("count", minimum=1), g.integer("keep", minimum=1)
        if experts % count or keep > count or top > keep * (experts // count):
            raise FormatError(f"{where}: top {top} of {experts} experts in {keep} of {count} groups")
        return RoutedExpertsSpec(
            hidden=self.width, intermediate=expert.integer("ff", minimum=1), n_experts=experts, top=top, router_bias=False,
            names=names(router=p + "router"), scoring="all", groups=count, keep_groups=keep,
            out_scale=router.number("scale", 1.0), activation="clamped", limit=expert.number("limit", positive=True),
            alpha=GATE_SLOPE, expert_names=names(gate=p + "e{e}.gate", up=p + "e{e}.up", down=p + "e{e}.down"))

    def _norm(self, name: str):
        return NormSpec(self.width, self.eps, name)

    def model_spec(self) -> ModelSpec:
        layers = [json.loads(text) for text in self.layers]
        blocks, schedule = [], []
        for i, layer in enumerate(layers):
            where = f"config.json: layers[{i}]"
            if not isinstance(layer, dict):
                raise FormatError(f"{where} is not an object")
            raw, kind, p = layer.get("mixer"), layer.get("type"), f"l{i}."
            if not isinstance(raw, dict):
                raise FormatError(f"{where}: 'mixer' must be an object")
            cache_of = None
            if kind == "lightning":
                mixer = self._recurrence(p + "mix.", raw, f"{where}.mixer")
            elif kind == "latent_attention":
                mixer = self._latent(p + "mix.", raw, f"{where}.mixer")
            elif kind == "attention":
                source = None
                if raw.get("kv_from") is not None:
                    cache_of = ConfigReader(raw, f"{where}.mixer").integer("kv_from", minimum=0)
                    source = layers[cache_of].get("mixer") if cache_of < i and layers[cache_of].get("type") == "attention" else None
                    if not isinstance(source, dict) or source.get("kv_from") is not None:
                        raise FormatError(f"{where}: kv_from {cache_of} is no earlier attention layer with keys of its own")
                mixer = self._attention(p + "mix.", raw, f"{where}.mixer", source)
            else:
                raise Unsupported(f"{where}: a layer of type '{kind}' (built: 'lightning', 'attention', 'latent_attention')")
            mlp = layer.get("mlp")
            ffn = self._feed_forward(p + "mlp.", mlp, f"{where}.mlp") if mlp is not None else None
            norms = dict(mixer_norm=self._norm(p + "norm1"), ffn_norm=self._norm(p + "norm2") if ffn is not None else None)
            if self.streams is None:
                blocks.append(BlockSpec(mixer=mixer, feed_forward=ffn, **norms))
            else:
                def streams(q):
                    return names(**{role: f"{p}hc{q}.{role}" for role in ("in", "mix", "out")})
                blocks.append(StreamsBlockSpec(n_streams=self.streams, mixer=mixer, mixer_streams=streams(1), feed_forward=ffn,
                                               ffn_streams=streams(2) if ffn is not None else None, **norms))
            schedule.append(ScheduleEntry(i, cache_of=cache_of))
        return ModelSpec(
            architecture=self.architecture, vocab=self.vocab, hidden=self.width, max_positions=MAX_POSITIONS,
            embedding="embed", blocks=tuple(blocks), schedule=tuple(schedule), final_norm=self._norm("final.norm"),
            head="head", streams=self.streams or 0)
