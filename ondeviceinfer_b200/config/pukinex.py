"""Typed configuration of the Pukinex decoder, read from its own ``config.json`` keys.

``config.json`` holds ``vocab``, ``width``, ``norm.eps``, ``embedding.scale``, ``residual_mult``, ``streams``,
``logit_scale``, ``logit_softcap``, ``loop`` (``start``, ``stop``, ``times``) and a list ``layers``; each entry has
``type`` (``attention`` or ``parallel``), the mixer's sizes and constants under ``mixer`` and its feed-forward under
``mlp`` (null: none).

* ``attention``: ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``, ``softcap``; ``rot`` (``base``, ``dims``,
  optionally ``scaling.factor``, which divides every frequency) rotates pairs of neighbouring lanes; a head's value is
  its key before the rotation; the softmax has a sink; a sigmoid gate with one number per head multiplies the output.
* ``parallel``: two mixers on the same input, ``left_scale`` * left + ``right_scale`` * right.  ``left``: grouped
  attention (``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``) with biased projections, an RMS norm per query and
  key head, queries multiplied by a slowly growing number (``q_temp.coef``, ``q_temp.every``), a learned bias by distance
  (``bias_max``; the stored table's shape gives the number of its rows, ``bias_rows`` where there is no table yet), a
  sink and a sigmoid gate per lane.  ``right``: retention (``heads``, ``dim``, ``vdim``, ``rot``, ``decay``: one number
  per head).
* ``mlp.kind`` ``dense``: down(max(up x, 0)^2), ``ff`` lanes.

Norms are layer norms with weight and bias.  With ``streams`` s every sublayer reads a weighted sum of s residual streams
and mixes them anew; the final norm reads their sum.  Layers ``loop.start`` .. ``loop.stop`` - 1 run ``loop.times`` times
in a row with the same tensors, each pass on a cache of its own.  A key that is absent switches its mechanism off.
Tensor names: ``embed``, ``l<i>.norm1|norm2`` (``.b``), ``l<i>.hc1|hc2.in|out|mix``, ``l<i>.mix.*`` (``left.``,
``right.``), ``l<i>.mlp.up|down``, ``final.norm`` (``.b``), ``head``.
"""

from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, List, Mapping, Optional, Tuple

from .specs import (CappedAttentionSpec, EmbeddingSpec, HeadSpec, LayerNormSpec, MLPSpec, ModelPlan, NoPositionSpec, OrderEntry,
                    RetentionSpec, RotarySpec, SideBySideMixersSpec, StreamMixBlockSpec, names)

MIXERS = ("attention", "parallel")
FEED_FORWARDS = ("dense",)
ACTIVATION = "relu2"            # fixed by the design: the square of max(x, 0)
BIAS_ROWS = 32                  # rows of a distance table when neither a checkpoint nor the configuration says


def _need(raw: Mapping[str, Any], key: str, where: str):
    if not isinstance(raw, Mapping) or key not in raw:
        raise KeyError(f"config.json: {where} lacks {key!r}")
    return raw[key]


@dataclass(frozen=True)
class PukinexConfig:
    vocab_size: int
    hidden_size: int
    norm_eps: float
    layers: Tuple[Mapping[str, Any], ...]     # the entries of config.json["layers"], as read
    loop: Optional[Tuple[int, int, int]] = None       # (start, stop, times)
    embedding_scale: float = 1.0
    residual_mult: float = 1.0
    streams: Optional[int] = None             # None: one stream with the plain residual sum
    logit_scale: float = 1.0
    logit_softcap: Optional[float] = None

    architecture = "Pukinex"

    # ------------------------------------------------------------------ construction

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any]) -> "PukinexConfig":
        layers = _need(raw, "layers", "the model")
        if not isinstance(layers, list) or not layers:
            raise ValueError("config.json: 'layers' must be a non-empty list")
        loop = raw.get("loop")
        if loop is not None:
            loop = tuple(int(_need(loop, key, "loop")) for key in ("start", "stop", "times"))
        cap, streams = raw.get("logit_softcap"), raw.get("streams")
        config = cls(vocab_size=int(_need(raw, "vocab", "the model")), hidden_size=int(_need(raw, "width", "the model")),
                     norm_eps=float(_need(_need(raw, "norm", "the model"), "eps", "norm")),
                     layers=tuple(copy.deepcopy(layer) for layer in layers), loop=loop,
                     embedding_scale=float((raw.get("embedding") or {}).get("scale", 1.0)),
                     residual_mult=float(raw.get("residual_mult", 1.0)), streams=None if streams is None else int(streams),
                     logit_scale=float(raw.get("logit_scale", 1.0)), logit_softcap=None if cap is None else float(cap))
        config.validate()
        return config

    def to_dict(self) -> dict:
        out = {"architecture": self.architecture, "embedding": {"scale": self.embedding_scale},
               "layers": [copy.deepcopy(dict(layer)) for layer in self.layers], "logit_scale": self.logit_scale,
               "norm": {"eps": self.norm_eps}, "residual_mult": self.residual_mult, "vocab": self.vocab_size,
               "width": self.hidden_size}
        if self.loop is not None:
            out["loop"] = dict(zip(("start", "stop", "times"), self.loop))
        if self.streams is not None:
            out["streams"] = self.streams
        if self.logit_softcap is not None:
            out["logit_softcap"] = self.logit_softcap
        return out

    def validate(self) -> None:
        if self.vocab_size <= 0 or self.hidden_size <= 0 or self.norm_eps <= 0:
            raise ValueError("vocab, width and norm.eps must be positive")
        if self.streams is not None and self.streams <= 0:
            raise ValueError("streams must be positive")
        if self.logit_softcap is not None and self.logit_softcap <= 0:
            raise ValueError("logit_softcap must be positive")
        for i, layer in enumerate(self.layers):
            if layer.get("type") not in MIXERS:
                raise ValueError(f"layers[{i}].type is {layer.get('type')!r}; known: {MIXERS}")
            f = layer.get("mlp")
            if f is not None and f.get("kind") not in FEED_FORWARDS:
                raise ValueError(f"layers[{i}].mlp.kind is {f.get('kind')!r}; known: {FEED_FORWARDS}")
            m = _need(layer, "mixer", f"layers[{i}]")
            if layer["type"] == "parallel":
                for side in ("left", "right"):
                    _need(m, side, f"layers[{i}].mixer")
        if self.loop is not None:
            start, stop, times = self.loop
            if not 0 <= start < stop <= len(self.layers) or times < 1:
                raise ValueError(f"loop {self.loop}: 0 <= start < stop <= {len(self.layers)} layers and times >= 1")

    @property
    def stop_token_ids(self) -> tuple:
        return ()

    # ------------------------------------------------------------------ the plan

    def _norm(self, name: str, **kwargs) -> LayerNormSpec:
        return LayerNormSpec(self.hidden_size, self.norm_eps, name, name + ".b", **kwargs)

    @staticmethod
    def _position(m: Mapping[str, Any], dim: int, where: str, interleaved: bool):
        rot = m.get("rot")
        if not rot or not int(_need(rot, "dims", where)):
            return NoPositionSpec()
        factor = (rot.get("scaling") or {}).get("factor", 1.0)
        return RotarySpec(head_dim=dim, theta=float(_need(rot, "base", where)), rotary_dim=int(rot["dims"]),
                          interleaved=interleaved, linear_factor=float(factor))

    def _heads(self, m: Mapping[str, Any], where: str) -> dict:
        heads, dim = int(_need(m, "heads", where)), int(_need(m, "dim", where))
        return dict(hidden_size=self.hidden_size, num_heads=heads, num_kv_heads=int(m.get("kv_heads", heads)), head_dim=dim,
                    value_dim=int(m.get("vdim", dim)), scale=float(_need(m, "scale", where)))

    def _attention(self, m: Mapping[str, Any], where: str, p: str) -> CappedAttentionSpec:
        cap = m.get("softcap")
        return CappedAttentionSpec(
            **self._heads(m, where), position=self._position(m, int(m["dim"]), where + ".rot", interleaved=True), prefix=p,
            names=names(q="q", k="k", g="g", o="o"), softcap=None if cap is None else float(cap), sink=True,
            values_are_keys=True, gate="head")

    def _left(self, m: Mapping[str, Any], where: str, p: str, rows: Optional[int]) -> CappedAttentionSpec:
        warm = m.get("q_temp")
        if warm is not None:
            warm = (float(_need(warm, "coef", where + ".q_temp")), int(_need(warm, "every", where + ".q_temp")))
        return CappedAttentionSpec(
            **self._heads(m, where), position=NoPositionSpec(), prefix=p,
            names=names(q="q", k="k", v="v", o="o", g="g", q_bias="q.b", k_bias="k.b", v_bias="v.b", q_norm="q.norm",
                        k_norm="k.norm", rel="rel"),
            unit_norm_eps=self.norm_eps, sink=True, gate="lane", q_temperature=warm,
            bias_rows=int(m.get("bias_rows", BIAS_ROWS)) if rows is None else rows,
            bias_reach=float(_need(m, "bias_max", where)))

    def _right(self, m: Mapping[str, Any], where: str, p: str) -> RetentionSpec:
        dim = int(_need(m, "dim", where))
        return RetentionSpec(
            hidden_size=self.hidden_size, num_heads=int(_need(m, "heads", where)), qk_dim=dim, v_dim=int(m.get("vdim", dim)),
            decay=tuple(float(v) for v in _need(m, "decay", where)),
            position=self._position(m, dim, where + ".rot", interleaved=False), prefix=p,
            names=names(q="q", k="k", v="v", g="g", o="o"), norm_eps=self.norm_eps)

    def _mixer(self, i: int, layer: Mapping[str, Any], stored: Mapping[str, Any]):
        m, where, p = layer["mixer"], f"layers[{i}].mixer", f"l{i}.mix."
        if layer["type"] == "attention":
            return self._attention(m, where, p)
        table = stored.get(p + "left.rel")
        return SideBySideMixersSpec(
            left=self._left(m["left"], where + ".left", p + "left.", None if table is None else int(table.shape[0])),
            right=self._right(m["right"], where + ".right", p + "right."),
            left_scale=float(m.get("left_scale", 1.0)), right_scale=float(m.get("right_scale", 1.0)))

    def _mlp(self, i: int, layer: Mapping[str, Any]) -> Optional[MLPSpec]:
        f = layer.get("mlp")
        if f is None:
            return None
        return MLPSpec(self.hidden_size, int(_need(f, "ff", f"layers[{i}].mlp")), ACTIVATION, f"l{i}.mlp.",
                       names(up="up", down="down"))

    def layer_runs(self) -> List[int]:
        """The layers in the order in which they run."""
        n = len(self.layers)
        if self.loop is None:
            return list(range(n))
        start, stop, times = self.loop
        return list(range(start)) + list(range(start, stop)) * times + list(range(stop, n))

    def plan_for(self, stored: Mapping[str, Any]) -> ModelPlan:
        """The plan with the sizes that only the checkpoint's tensors give (the rows of the distance tables)."""
        layers: List[StreamMixBlockSpec] = []
        ignored: List[str] = []
        streams = self.streams or 1
        # one stream may come without coefficients: the plain residual sum
        plain = self.streams is None or (self.streams == 1 and bool(stored) and not any(".hc1." in name for name in stored))
        mix = lambda i, q: None if plain else tuple(f"l{i}.hc{q}.{role}" for role in ("in", "out", "mix"))
        for i, layer in enumerate(self.layers):
            mlp = self._mlp(i, layer)
            has = mlp is not None
            layers.append(StreamMixBlockSpec(
                mixer_norm=self._norm(f"l{i}.norm1"), mixer=self._mixer(i, layer, stored),
                ffn_norm=self._norm(f"l{i}.norm2") if has else None, ffn=mlp, hidden_size=self.hidden_size, streams=streams,
                residual_mult=self.residual_mult, mixer_names=mix(i, 1), ffn_names=mix(i, 2) if has else None))
            if not has:       # a layer without a feed-forward may still store what belongs to one
                ignored += [f"l{i}.norm2", f"l{i}.norm2.b"] + [f"l{i}.hc2.{role}" for role in ("in", "out", "mix")]
        plan = ModelPlan(
            embedding=EmbeddingSpec(self.vocab_size, self.hidden_size, "embed", scale=self.embedding_scale, streams=streams),
            layers=tuple(layers), order=tuple(OrderEntry(layer=i) for i in self.layer_runs()),
            final_norm=self._norm("final.norm", streams=streams, output_scale=self.logit_scale),
            head=HeadSpec(self.vocab_size, self.hidden_size, "head", softcap=self.logit_softcap),
            ignored_tensors=tuple(ignored))
        plan.validate()
        return plan

    def to_plan(self) -> ModelPlan:
        return self.plan_for({})
