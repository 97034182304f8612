"""Configuration of the Duvozen decoder, read from its own config.json keys.

A Duvozen model is a list of layers with norms on the parts' results only:
x += norm1(mixer(c1(x))); x += norm2(feed_forward(c2(x))), layer norms with a weight and no bias, where
c(x) = x + conv(x) adds a short causal convolution of the stream (`canon.taps` taps per channel) to what a part
reads. A layer's `type` names its mixer: `hgrn2` (a linear recurrence whose forget gate decides what is written),
`latent_attention` (attention over one cached latent row with a rotated key part that all heads share) or
`attention` (grouped softmax attention with a norm per head, a learned sink per head and an element-wise gate).
Its `mlp` is `dense` (gated, tanh-form gelu), `moe` (routed experts: sigmoid scores, the weight on an expert's
input, and a shared expert) or null. The embedding and the logits are scaled; the head is a matrix of its own.
"""
from __future__ import annotations

import json
from dataclasses import dataclass

from ..errors import FormatError, Unsupported
from ..parts.spec import (ForgetRecurrenceSpec, GatedAttentionSpec, GatedMlpSpec, LayerNormSpec, ModelSpec,
                          OutputNormBlockSpec, PositionSpec, RotaryLatentSpec, RoutedExpertsSpec, ScheduleEntry, names)
from .base import ConfigReader

# no key of the configuration bounds a sequence: the engine's context does
MAX_POSITIONS = 1 << 22


@dataclass(frozen=True)
class DuvozenConfig:
    """`layers` keeps the configuration's list as JSON text per layer (hashable); the typed view is `model_spec()`."""
    vocab: int
    width: int
    eps: float
    embedding_scale: float
    logit_scale: float
    taps: int
    layers: tuple

    architecture = "Duvozen"

    @classmethod
    def from_dict(cls, raw: dict, where: str = "config.json") -> "DuvozenConfig":
        r = ConfigReader(raw, where)
        layers = raw.get("layers")
        if not isinstance(layers, list) or not layers:
            raise FormatError(f"{where}: 'layers' must be a non-empty list")
        norm = ConfigReader(r.mapping("norm"), f"{where}: norm")
        embedding, canon = r.mapping("embedding", None), r.mapping("canon", None)
        scale = ConfigReader(embedding, f"{where}: embedding").number("scale", 1.0) if embedding is not None else 1.0
        taps = ConfigReader(canon, f"{where}: canon").integer("taps", minimum=1) if canon is not None else 0
        config = cls(vocab=r.integer("vocab", minimum=1), width=r.integer("width", minimum=1),
                     eps=norm.number("eps", positive=True), embedding_scale=scale,
                     logit_scale=r.number("logit_scale", 1.0), taps=taps,
                     layers=tuple(json.dumps(layer, sort_keys=True) for layer in layers))
        config.model_spec()            # every layer is read once here, so that a bad key is reported at load
        return config

    def to_dict(self) -> dict:
        out = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
               "norm": {"eps": self.eps}, "embedding": {"scale": self.embedding_scale}, "logit_scale": self.logit_scale,
               "layers": [json.loads(text) for text in self.layers]}
        if self.taps:
            out["canon"] = {"taps": self.taps}
        return out

    def to_json(self) -> str:
        return json.dumps(self.to_dict(), indent=2) + "\n"

    # ------------------------------------------------------------------ the model as data

    @staticmethod
    def _position(m, unit: int, pairing: str, where: str):
        """The rotation of units of `unit` elements (None: a mixer without one)."""
        rot = m.mapping("rot", None)
        if rot is None:
            return None
        rr = ConfigReader(rot, f"{where}: rot")
        dims = rr.integer("dims", minimum=2)
        if dims % 2 or dims > unit:
            raise FormatError(f"{where}: rot.dims {dims} must be even and at most {unit}")
        scaling = None
        sc = rr.mapping("scaling", None)
        if sc is not None:
            ss = ConfigReader(sc, f"{where}: rot.scaling")
            scaling = tuple(sorted({"type": "ramp", "factor": ss.number("factor", positive=True),
                                    "original": ss.number("original", positive=True),
                                    "fast": ss.number("fast", positive=True),
                                    "slow": ss.number("slow", positive=True)}.items()))
        return PositionSpec(head_dim=unit, theta=rr.number("base", positive=True), max_positions=MAX_POSITIONS,
                            scaling=scaling, pairing=pairing, rotary_dim=dims)

    def _attention(self, p: str, raw: dict, where: str):
        m = ConfigReader(raw, where)
        heads, kv_heads = m.integer("heads", minimum=1), m.integer("kv_heads", minimum=1)
        if heads % kv_heads:
            raise FormatError(f"{where}: {heads} heads are no multiple of {kv_heads} kv_heads")
        dim = m.integer("dim", minimum=1)
        return GatedAttentionSpec(
            hidden=self.width, n_heads=heads, n_kv_heads=kv_heads, head_dim=dim,
            value_dim=m.integer("vdim", dim, minimum=1), scale=m.number("scale"), window=0, values_are_keys=False,
            out_gate=True, position=self._position(m, dim, "half", where), head_norm=True, norm_eps=self.eps, sink=True,
            names=names(q=p + "q", k=p + "k", v=p + "v", o=p + "o", gate=p + "g", sink=p + "sink", q_norm=p + "q.norm",
                        k_norm=p + "k.norm"))

    def _latent(self, p: str, raw: dict, where: str):
        m = ConfigReader(raw, where)
        rot_dim = m.integer("rot_dim", minimum=1)
        return RotaryLatentSpec(
            hidden=self.width, n_heads=m.integer("heads", minimum=1), head_dim=m.integer("dim", minimum=1),
            rot_dim=rot_dim, value_dim=m.integer("vdim", minimum=1), kv_rank=m.integer("kv_rank", minimum=1),
            scale=m.number("scale"), eps=self.eps, position=self._position(m, rot_dim, "interleaved", where),
            names=names(q=p + "q", dkv=p + "dkv", dkv_norm=p + "dkv.norm", uk=p + "uk", uv=p + "uv", o=p + "o"))

    def _recurrence(self, p: str, raw: dict, where: str):
        m = ConfigReader(raw, where)
        return ForgetRecurrenceSpec(
            hidden=self.width, n_heads=m.integer("heads", minimum=1), head_dim=m.integer("dim", minimum=1),
            value_dim=m.integer("vdim", minimum=1), eps=self.eps,
            names=names(q=p + "q", f=p + "f", f_bias=p + "f.b", lower=p + "lower", v=p + "v", norm=p + "norm", o=p + "o"))

    def _feed_forward(self, p: str, raw: dict, where: str):
        f = ConfigReader(raw, where)
        kind = f.string("kind", "dense")
        if kind == "dense":
            return GatedMlpSpec(hidden=self.width, intermediate=f.integer("ff", minimum=1), activation="gelu_tanh",
                                names=names(gate=p + "gate", up=p + "up", down=p + "down"))
        if kind == "moe":
            router = ConfigReader(f.mapping("router"), f"{where}: router")
            expert = ConfigReader(f.mapping("expert"), f"{where}: expert")
            experts, top = router.integer("experts", minimum=1), router.integer("top", minimum=1)
            if top > experts:
                raise FormatError(f"{where}: top {top} of {experts} experts")
            shared, raw_shared = None, f.mapping("shared", None)
            if raw_shared is not None:
                shared = GatedMlpSpec(hidden=self.width, activation="silu",
                                      intermediate=ConfigReader(raw_shared, f"{where}: shared").integer("ff", minimum=1),
                                      names=names(gate=p + "shared.gate", up=p + "shared.up", down=p + "shared.down"))
            return RoutedExpertsSpec(
                hidden=self.width, intermediate=expert.integer("ff", minimum=1), n_experts=experts, top=top,
                router_bias=False, names=names(router=p + "router"), scoring="sigmoid", weight_on_input=True, shared=shared,
                expert_names=names(gate=p + "e{e}.gate", up=p + "e{e}.up", down=p + "e{e}.down"))
        raise Unsupported(f"{where}: kind '{kind}' (built: 'dense', 'moe')")

    def _norm(self, name: str):
        return LayerNormSpec(self.width, self.eps, name)

    def model_spec(self) -> ModelSpec:
        mixers = {"hgrn2": self._recurrence, "latent_attention": self._latent, "attention": self._attention}
        blocks = []
        for i, text in enumerate(self.layers):
            layer = json.loads(text)
            where = f"config.json: layers[{i}]"
            if not isinstance(layer, dict):
                raise FormatError(f"{where} is not an object")
            if not isinstance(layer.get("mixer"), dict):
                raise FormatError(f"{where}: 'mixer' must be an object")
            if layer.get("type") not in mixers:
                raise Unsupported(f"{where}: a layer of type '{layer.get('type')}' (built: {', '.join(map(repr, mixers))})")
            mixer = mixers[layer["type"]](f"l{i}.mix.", layer["mixer"], f"{where}.mixer")
            mlp = layer.get("mlp")
            ffn = self._feed_forward(f"l{i}.mlp.", mlp, f"{where}.mlp") if mlp is not None else None
            blocks.append(OutputNormBlockSpec(
                mixer=mixer, mixer_norm=self._norm(f"l{i}.norm1"), feed_forward=ffn,
                ffn_norm=self._norm(f"l{i}.norm2") if ffn is not None else None, conv_taps=self.taps,
                mixer_conv=f"l{i}.canon1" if self.taps else None,
                ffn_conv=f"l{i}.canon2" if self.taps and ffn is not None else None))
        return ModelSpec(
            architecture=self.architecture, vocab=self.vocab, hidden=self.width, max_positions=MAX_POSITIONS,
            embedding="embed", blocks=tuple(blocks), schedule=tuple(ScheduleEntry(i) for i in range(len(blocks))),
            final_norm=self._norm("final.norm"), head="head", embedding_scale=self.embedding_scale,
            logit_scale=self.logit_scale)
