"""Typed configuration of the Vumedra decoder, read from its config.json.

config.json carries ``architecture``, ``width``, ``vocab``, ``norm.eps``, ``embedding.bigram`` (``buckets``, ``mul_prev``,
``mul_cur``) and ``layers``: one entry per layer with ``type`` (``attention``, ``mlstm`` or ``rglru``), the mixer's sizes and
constants under ``mixer``, and the feed-forward under ``mlp`` (``{"kind": "dense", "ff": n}``, ``{"kind": "moe", "expert":
{"ff": n}, "router": {"experts": e, "top": k}, "shared": {"ff": n}}`` or null).
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping

LAYER_TYPES = ("attention", "mlstm", "rglru")
MLP_KINDS = ("dense", "moe")


@dataclass(frozen=True)
class VumedraLayer:
    type: str
    mixer: Mapping[str, Any]
    mlp: Mapping[str, Any] | None  # None: no feed-forward


@dataclass(frozen=True)
class VumedraConfig:
    width: int
    vocab: int
    eps: float
    bigram: Mapping[str, Any] | None  # None: no second table in the embedding
    layers: tuple[VumedraLayer, ...]
    raw: Mapping[str, Any]

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any]) -> "VumedraConfig":
        missing = [k for k in ("width", "vocab", "layers", "norm") if k not in raw]
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
            layers.append(VumedraLayer(kind, entry["mixer"], mlp))
        cfg = cls(width=int(raw["width"]), vocab=int(raw["vocab"]), eps=float(raw["norm"]["eps"]),
                  bigram=(raw.get("embedding") or {}).get("bigram"), layers=tuple(layers), raw=raw)
        cfg.validate()
        return cfg

    def validate(self) -> None:
        if self.width < 1 or self.vocab < 1 or not self.layers:
            raise ValueError("width, vocab and the number of layers must be positive")
        if self.bigram is not None and int(self.bigram["buckets"]) < 1:
            raise ValueError(f"embedding.bigram.buckets={self.bigram['buckets']} must be positive")
        sizes = {"attention": ("heads", "kv_heads", "dim", "vdim"), "mlstm": ("heads", "dim", "vdim"), "rglru": ("width", "blocks", "conv")}
        for i, layer in enumerate(self.layers):
            m = layer.mixer
            for key in sizes[layer.type]:
                if int(m[key]) < 1:
                    raise ValueError(f"layer {i}: {key}={m[key]} must be positive")
            if layer.type == "attention":
                if int(m["heads"]) % int(m["kv_heads"]):
                    raise ValueError(f"layer {i}: {m['heads']} query heads are not a multiple of {m['kv_heads']} key/value heads")
                if m.get("q_temp") is not None and float(m["q_temp"]["every"]) <= 0:
                    raise ValueError(f"layer {i}: q_temp.every={m['q_temp']['every']} must be positive")
            elif layer.type == "mlstm":
                if float(m["gate_cap"]) <= 0:
                    raise ValueError(f"layer {i}: gate_cap={m['gate_cap']} must be positive")
            elif int(m["width"]) % int(m["blocks"]):
                raise ValueError(f"layer {i}: {m['width']} channels do not split into {m['blocks']} equal parts")
            mlp = layer.mlp
            if mlp is not None and mlp["kind"] == "moe":
                r = mlp["router"]
                if not 1 <= int(r["top"]) <= int(r["experts"]):
                    raise ValueError(f"layer {i}: top={r['top']} of {r['experts']} experts")
