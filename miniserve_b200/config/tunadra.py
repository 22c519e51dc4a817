"""Typed configuration of the Tunadra decoder, read from its config.json.

config.json carries ``architecture``, ``width``, ``vocab``, ``norm.eps``, ``embedding.scale``, ``streams``, ``logit_softcap`` and
``layers``: one entry per layer with ``type`` (``attention`` or ``wkv``), the mixer's sizes and constants under ``mixer``, and the
feed-forward under ``mlp`` (null, or ``{"kind": "moe", "expert": {"ff": n, "limit": c}, "router": {"experts": e, "top": k, "groups":
{"count": g, "keep": m}, "scale": s}, "shared": {"ff": n, "limit": c}}``). The rank of the decays' projection is read off the
checkpoint's tensor shapes (``complete_from_shapes``), or given as ``decay_rank`` in a mixer's entry.
"""

from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, Mapping

LAYER_TYPES = ("attention", "wkv")
MLP_KINDS = ("moe",)


@dataclass(frozen=True)
class TunadraLayer:
    type: str
    mixer: Mapping[str, Any]
    mlp: Mapping[str, Any] | None  # None: no feed-forward


@dataclass(frozen=True)
class TunadraConfig:
    width: int
    vocab: int
    eps: float
    embedding_scale: float
    streams: int
    logit_softcap: float
    layers: tuple[TunadraLayer, ...]
    raw: Mapping[str, Any]

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any]) -> "TunadraConfig":
        missing = [k for k in ("width", "vocab", "layers", "norm", "streams", "logit_softcap") if k not in raw]
        if missing:
            raise KeyError(f"config.json lacks {missing}")
        layers = []
        for i, entry in enumerate(raw["layers"]):
            kind = entry.get("type")
            if kind not in LAYER_TYPES:
                raise NotImplementedError(f"layer {i}: type {kind!r} is not one of {LAYER_TYPES}")
            mlp = entry.get("mlp")
            if mlp is not None and mlp.get("kind") not in MLP_KINDS:
                raise NotImplementedError(f"layer {i}: feed-forward kind {mlp.get('kind')!r} is not one of {MLP_KINDS}")
            layers.append(TunadraLayer(kind, entry["mixer"], mlp))
        cfg = cls(width=int(raw["width"]), vocab=int(raw["vocab"]), eps=float(raw["norm"]["eps"]),
                  embedding_scale=float((raw.get("embedding") or {}).get("scale", 1.0)), streams=int(raw["streams"]),
                  logit_softcap=float(raw["logit_softcap"]), layers=tuple(layers), raw=raw)
        cfg.validate()
        return cfg

    def validate(self) -> None:
        if self.width < 1 or self.vocab < 1 or not self.layers:
            raise ValueError("width, vocab and the number of layers must be positive")
        if self.streams < 1:
            raise ValueError(f"streams={self.streams} must be positive")
        if self.logit_softcap <= 0:
            raise ValueError(f"logit_softcap={self.logit_softcap} must be positive")
        sizes = {"attention": ("heads", "kv_heads", "dim", "vdim"), "wkv": ("heads", "dim")}
        shared_values = None
        for i, layer in enumerate(self.layers):
            m = layer.mixer
            for key in sizes[layer.type]:
                if int(m[key]) < 1:
                    raise ValueError(f"layer {i}: {key}={m[key]} must be positive")
            if layer.type == "attention":
                if int(m["heads"]) % int(m["kv_heads"]):
                    raise ValueError(f"layer {i}: {m['heads']} query heads are not a multiple of {m['kv_heads']} key/value heads")
                if m.get("v_mix"):
                    width = int(m["kv_heads"]) * int(m["vdim"])
                    if shared_values is not None and shared_values[1] != width:
                        raise ValueError(f"layer {i}: values of {width} numbers cannot be mixed with layer {shared_values[0]}'s {shared_values[1]}")
                    shared_values = shared_values or (i, width)
            elif "decay_rank" not in m:
                raise KeyError(f"layer {i}: the rank of the decays' projection is unknown (no checkpoint, no 'decay_rank')")
            mlp = layer.mlp
            if mlp is not None:
                r = mlp["router"]
                groups = r.get("groups") or {"count": 1, "keep": 1}
                experts, count, keep = int(r["experts"]), int(groups["count"]), int(groups["keep"])
                if not 1 <= int(r["top"]) <= experts:
                    raise ValueError(f"layer {i}: top={r['top']} of {experts} experts")
                if count < 1 or experts % count or not 1 <= keep <= count or keep * (experts // count) < int(r["top"]):
                    raise ValueError(f"layer {i}: {experts} experts in {count} groups of which {keep} are kept cannot give {r['top']} choices")
                for part in ("expert", "shared"):
                    if mlp.get(part) and float(mlp[part]["limit"]) < 0:
                        raise ValueError(f"layer {i}: {part}.limit={mlp[part]['limit']} must not be negative")


def complete_from_shapes(raw: Mapping[str, Any], shapes: Mapping[str, tuple]) -> dict[str, Any]:
    """The ranks of the decays' low-rank projections, read off the checkpoint's tensor shapes."""
    raw = copy.deepcopy(dict(raw))
    for i, entry in enumerate(raw.get("layers", [])):
        name = f"l{i}.mix.w1"
        if entry.get("type") == "wkv" and "decay_rank" not in entry.get("mixer", {}) and name in shapes:
            entry["mixer"]["decay_rank"] = int(shapes[name][0])
    return raw
