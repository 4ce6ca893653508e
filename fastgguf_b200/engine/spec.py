"""The data that describes a model, as Python objects: which parts, in which layers, run in which order.

The host works from the JSON form (``csrc/fastgguf_parts.h`` describes it); these classes build and read it:

* every part is a :class:`PartSpec` - a registered kind name, its sizes and constants as parameters, and
  the checkpoint names of its tensors;
* every layer names its own block arrangement, mixer, feed-forward and norms, so one model can mix kinds
  layer by layer;
* the order in which layers run is the list ``schedule``: an entry may name a layer that already ran (shared
  weights, a cache of its own) or read the cache of an earlier entry instead of writing one.

The reference expresses the same choices as flags and optional per-layer tensors on one struct (``is_swa[]``,
``kv_donor[]``, optional norms; fastgguf.c:4064-4100) and a fixed ``for il < n_layer`` loop (:4674).
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Dict, List, Optional, Tuple


@dataclass
class PartSpec:
    """A part to build: ``kind`` is looked up in the part registry of its role."""

    kind: str
    params: dict = field(default_factory=dict)
    #: local tensor name of the part -> tensor name in the checkpoint
    tensors: Dict[str, str] = field(default_factory=dict)

    def to_json(self) -> dict:
        def conv(v):
            return v.to_json() if isinstance(v, PartSpec) else v
        return {"kind": self.kind, "params": {k: conv(v) for k, v in self.params.items()}, "tensors": dict(self.tensors)}

    @classmethod
    def from_json(cls, j: dict) -> "PartSpec":
        params = {k: (cls.from_json(v) if isinstance(v, dict) and "kind" in v and "params" in v else v)
                  for k, v in (j.get("params") or {}).items()}
        return cls(j["kind"], params, dict(j.get("tensors") or {}))


@dataclass
class LayerSpec:
    block: str                     # arrangement kind, e.g. "prenorm", "sandwich"
    mixer: PartSpec
    feed_forward: Optional[PartSpec]           # None: a layer of a mixer alone
    mixer_norm: Optional[PartSpec]             # None: block "postnorm", whose sublayers read the stream itself
    feed_forward_norm: Optional[PartSpec]
    #: norms on a sublayer's output, before it joins the residual stream (block "sandwich")
    mixer_post_norm: Optional[PartSpec] = None
    feed_forward_post_norm: Optional[PartSpec] = None
    #: what the layer adds to the stream from its tokens, behind its sublayers (role ``token_input``)
    token_input: Optional[PartSpec] = None

    def to_json(self) -> dict:
        def opt(p):
            return p.to_json() if p is not None else None
        j = {"block": self.block, "mixer": self.mixer.to_json(), "feed_forward": opt(self.feed_forward),
             "mixer_norm": opt(self.mixer_norm), "feed_forward_norm": opt(self.feed_forward_norm)}
        if self.mixer_post_norm is not None:
            j["mixer_post_norm"] = self.mixer_post_norm.to_json()
        if self.feed_forward_post_norm is not None:
            j["feed_forward_post_norm"] = self.feed_forward_post_norm.to_json()
        if self.token_input is not None:
            j["token_input"] = self.token_input.to_json()
        return j


@dataclass
class RunSpec:
    """One entry of the execution order."""

    layer: int
    #: index of an EARLIER schedule entry whose cache this run reads instead of owning one
    cache_from: Optional[int] = None
    #: the model's ``reentry`` map (stream and embedding output -> stream) runs in front of this entry
    reenter: bool = False
    #: with ``reenter``: the number of the pass that begins here
    pass_number: Optional[int] = None


@dataclass
class ModelSpec:
    hidden_size: int
    vocab_size: int
    max_positions: int
    embedding: PartSpec
    layers: List[LayerSpec]
    schedule: List[RunSpec]
    final_norm: PartSpec
    head: PartSpec
    stop_token_ids: Tuple[int, ...] = ()
    #: regular expressions of checkpoint tensors that may be present without being used
    ignored_tensors: Tuple[str, ...] = ()
    #: optional map of the residual stream that also reads the embedding's output (schedule entries ask for it)
    reentry: Optional[PartSpec] = None

    def to_json(self) -> dict:
        extra = {"reentry": self.reentry.to_json()} if self.reentry is not None else {}
        return {
            **extra,
            "hidden_size": self.hidden_size, "vocab_size": self.vocab_size, "max_positions": self.max_positions,
            "embedding": self.embedding.to_json(), "final_norm": self.final_norm.to_json(), "head": self.head.to_json(),
            "layers": [l.to_json() for l in self.layers],
            "schedule": [dict({"layer": r.layer, "cache_from": r.cache_from}, **({"reenter": True} if r.reenter else {}),
                          **({"pass": r.pass_number} if r.pass_number is not None else {})) for r in self.schedule],
            "stop_token_ids": list(self.stop_token_ids), "ignored_tensors": list(self.ignored_tensors),
        }

    @classmethod
    def from_json(cls, j: dict) -> "ModelSpec":
        P = PartSpec.from_json

        def O(v):
            return P(v) if v else None
        return cls(
            hidden_size=j["hidden_size"], vocab_size=j["vocab_size"], max_positions=j["max_positions"],
            embedding=P(j["embedding"]), final_norm=P(j["final_norm"]), head=P(j["head"]),
            layers=[LayerSpec(l["block"], P(l["mixer"]), O(l.get("feed_forward")), O(l.get("mixer_norm")), O(l.get("feed_forward_norm")),
                              O(l.get("mixer_post_norm")), O(l.get("feed_forward_post_norm")), O(l.get("token_input"))) for l in j["layers"]],
            schedule=[RunSpec(r["layer"], r.get("cache_from"), bool(r.get("reenter", False)), r.get("pass")) for r in j["schedule"]],
            reentry=O(j.get("reentry")),
            stop_token_ids=tuple(j.get("stop_token_ids") or ()), ignored_tensors=tuple(j.get("ignored_tensors") or ()),
        )
