"""Typed configuration of the Noganex decoder, read from its own ``config.json`` keys.

``config.json`` holds ``vocab``, ``width``, ``norm.eps``, ``logit_scale`` and a list ``layers``; each entry has ``type``
(``attention`` or ``delta``), the mixer's sizes and constants under ``mixer`` and its feed-forward under ``mlp`` (null:
none).

* ``attention``: ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``; RMS norms over a token's whole q and k rows;
  ``rot`` (``base``, ``dims``, optionally ``scaling`` with ``factor``, ``original``, ``fast``, ``slow``: frequencies slowed
  by a ramp over their index) rotates half-split pairs; the heads' scores are mixed by a stored matrix before the
  softmax; ``mask.size``: positions see their own chunk of that many.
* ``delta``: ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``conv``: a gated delta rule with one decay per head.
* ``mlp.kind`` ``dense``: tanh-GELU gate with biases (``ff``).  ``moe``: ``router.experts`` SiLU-gated experts of
  ``expert.ff`` lanes, ``router.top`` chosen by sigmoid scores plus a stored correction and weighted by the scores
  divided by their sum times ``router.scale``; ``shared.ff``: one more expert that every token takes.

A layer with ``weights_of``: j runs the tensors of layer j on a cache and a state of its own.  What a sublayer adds to
the stream is gated lane by lane by sigmoid(rg x + b) and then RMS-normed; the sublayers read the stream itself.  A key
that is absent switches its mechanism off.
Tensor names: ``embed``, ``l<i>.norm1|norm2|rg1|rg1.b|rg2|rg2.b``, ``l<i>.mix.*``, ``l<i>.mlp.*``, ``final.norm``, ``head``.
"""

from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, List, Mapping, Tuple

from .specs import (EmbeddingSpec, GatedMLPSpec, GatedPostNormBlockSpec, HeadDeltaSpec, HeadSpec, MixedAttentionSpec, ModelPlan,
                    NoPositionSpec, OrderEntry, RMSNormSpec, RotarySpec, RoutedExpertsSpec, names)

MIXERS = ("attention", "delta")
FEED_FORWARDS = ("dense", "moe")


def _need(raw: Mapping[str, Any], key: str, where: str):
    if not isinstance(raw, Mapping) or key not in raw:
        raise KeyError(f"config.json: {where} lacks {key!r}")
    return raw[key]


@dataclass(frozen=True)
class NoganexConfig:
    vocab_size: int
    hidden_size: int
    norm_eps: float
    layers: Tuple[Mapping[str, Any], ...]     # the entries of config.json["layers"], as read
    logit_scale: float = 1.0

    architecture = "Noganex"

    # ------------------------------------------------------------------ construction

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any]) -> "NoganexConfig":
        layers = _need(raw, "layers", "the model")
        if not isinstance(layers, list) or not layers:
            raise ValueError("config.json: 'layers' must be a non-empty list")
        config = cls(vocab_size=int(_need(raw, "vocab", "the model")), hidden_size=int(_need(raw, "width", "the model")),
                     norm_eps=float(_need(_need(raw, "norm", "the model"), "eps", "norm")),
                     layers=tuple(copy.deepcopy(layer) for layer in layers), logit_scale=float(raw.get("logit_scale", 1.0)))
        config.validate()
        return config

    def to_dict(self) -> dict:
        return {"architecture": self.architecture, "layers": [copy.deepcopy(dict(layer)) for layer in self.layers],
                "logit_scale": self.logit_scale, "norm": {"eps": self.norm_eps}, "vocab": self.vocab_size,
                "width": self.hidden_size}

    def validate(self) -> None:
        if self.vocab_size <= 0 or self.hidden_size <= 0 or self.norm_eps <= 0:
            raise ValueError("vocab, width and norm.eps must be positive")
        for i, layer in enumerate(self.layers):
            if layer.get("type") not in MIXERS:
                raise ValueError(f"layers[{i}].type is {layer.get('type')!r}; known: {MIXERS}")
            f = layer.get("mlp")
            if f is not None and f.get("kind") not in FEED_FORWARDS:
                raise ValueError(f"layers[{i}].mlp.kind is {f.get('kind')!r}; known: {FEED_FORWARDS}")
            owner = self.layers[self.owner_of(i)]
            if owner["type"] != layer["type"]:
                raise ValueError(f"layers[{i}] is of type {layer['type']!r} and uses the weights of a layer of type {owner['type']!r}")
            _need(owner, "mixer", f"layers[{self.owner_of(i)}]")

    def owner_of(self, i: int) -> int:
        """The layer whose tensors layer i uses."""
        seen = {i}
        while self.layers[i].get("weights_of") is not None:
            j = int(self.layers[i]["weights_of"])
            if not 0 <= j < len(self.layers) or j in seen:
                raise ValueError(f"layers[{i}].weights_of is {j}: no layer that has weights")
            seen.add(j)
            i = j
        return i

    @property
    def stop_token_ids(self) -> tuple:
        return ()

    # ------------------------------------------------------------------ the plan

    def _norm(self, name: str, output_scale: float = 1.0) -> RMSNormSpec:
        return RMSNormSpec(self.hidden_size, self.norm_eps, name, scale_in_fp32=True, output_scale=output_scale)

    @staticmethod
    def _position(m: Mapping[str, Any], dim: int, where: str):
        rot = m.get("rot")
        if not rot or not int(_need(rot, "dims", where)):
            return NoPositionSpec()
        scaling = rot.get("scaling")
        ramp = None if not scaling else tuple(float(_need(scaling, key, where + ".scaling"))
                                              for key in ("factor", "original", "fast", "slow"))
        return RotarySpec(head_dim=dim, theta=float(_need(rot, "base", where)), rotary_dim=int(rot["dims"]), index_ramp=ramp)

    def _mixer(self, i: int, layer: Mapping[str, Any]):
        m, where, p = layer["mixer"], f"layers[{i}].mixer", f"l{i}.mix."
        heads, dim = int(_need(m, "heads", where)), int(_need(m, "dim", where))
        kv_heads, value_dim = int(m.get("kv_heads", heads)), int(m.get("vdim", dim))
        if layer["type"] == "attention":
            size = (m.get("mask") or {}).get("size")
            return MixedAttentionSpec(
                hidden_size=self.hidden_size, num_heads=heads, num_kv_heads=kv_heads, head_dim=dim, value_dim=value_dim,
                scale=float(_need(m, "scale", where)), position=self._position(m, dim, where + ".rot"), prefix=p,
                names=names(q="q", k="k", v="v", o="o", q_norm="q.norm", k_norm="k.norm", talk="talk"),
                row_norm_eps=self.norm_eps, chunk=None if size is None else int(size))
        return HeadDeltaSpec(
            hidden_size=self.hidden_size, num_heads=heads, num_kv_heads=kv_heads, qk_dim=dim, v_dim=value_dim,
            conv_taps=int(_need(m, "conv", where)), norm_eps=self.norm_eps, prefix=p,
            names=names(q="q", k="k", v="v", q_conv="q.conv", k_conv="k.conv", v_conv="v.conv", b="b", A_log="A_log",
                        dt_bias="dt_bias", a="a", g="g", norm="norm", o="o"))

    def _mlp(self, i: int, layer: Mapping[str, Any]):
        f = layer.get("mlp")
        if f is None:
            return None
        where, p = f"layers[{i}].mlp", f"l{i}.mlp."
        if f["kind"] == "dense":
            return GatedMLPSpec(self.hidden_size, int(_need(f, "ff", where)), "gelu_tanh", p,
                                names(gate="gate", up="up", down="down", gate_bias="gate.b", up_bias="up.b", down_bias="down.b"))
        router, expert = _need(f, "router", where), _need(f, "expert", where)
        return RoutedExpertsSpec(
            hidden_size=self.hidden_size, expert_size=int(_need(expert, "ff", where + ".expert")),
            num_experts=int(_need(router, "experts", where + ".router")), num_identity=0,
            top_k=int(_need(router, "top", where + ".router")), num_groups=1, keep_groups=1, limit=0.0, prefix=p,
            has_correction=True, shared_size=int((f.get("shared") or {}).get("ff", 0)), scoring="sigmoid",
            expert_form="gated_silu", renormalise=True, weight_scale=float(router.get("scale", 1.0)))

    def to_plan(self) -> ModelPlan:
        layers: List[GatedPostNormBlockSpec] = []
        index_of = {}
        ignored: List[str] = []
        for i, layer in enumerate(self.layers):
            if self.owner_of(i) != i:
                continue
            mlp = self._mlp(i, layer)
            index_of[i] = len(layers)
            has = mlp is not None
            layers.append(GatedPostNormBlockSpec(
                mixer=self._mixer(i, layer), mixer_norm=self._norm(f"l{i}.norm1"), ffn=mlp,
                ffn_norm=self._norm(f"l{i}.norm2") if has else None, hidden_size=self.hidden_size,
                mixer_gate_name=f"l{i}.rg1", mixer_gate_bias_name=f"l{i}.rg1.b", ffn_gate_name=f"l{i}.rg2" if has else None,
                ffn_gate_bias_name=f"l{i}.rg2.b" if has else None))
            if not has:       # a layer without a feed-forward may still store what belongs to one
                ignored += [f"l{i}.norm2", f"l{i}.rg2", f"l{i}.rg2.b"]
        plan = ModelPlan(
            embedding=EmbeddingSpec(self.vocab_size, self.hidden_size, "embed"), layers=tuple(layers),
            order=tuple(OrderEntry(layer=index_of[self.owner_of(i)]) for i in range(len(self.layers))),
            final_norm=self._norm("final.norm", self.logit_scale), head=HeadSpec(self.vocab_size, self.hidden_size, "head"),
            ignored_tensors=tuple(ignored))
        plan.validate()
        return plan
