"""The Tunadra decoder as data: its configuration mapped onto parts.

The stream starts as the token's scaled row plus a sinusoidal vector of the position, in several equal copies (hyper-connections): every
sublayer reads the norm of a weighted sum of the streams, and its output changes all of them at once. Two mixers: ``attention``
(grouped heads with a key and a value size, queries and keys divided by their root mean square, no rotation, values mixed with those of
the first such layer, a gate per head) and ``wkv`` (RWKV-style time mixing behind a token shift: a decay per key channel and token, a
bonus for the token's own write). Feed-forward: a mixture of clamped gated experts, chosen by sigmoid scores within the best groups and
weighed by the renormalised scores, beside a shared expert; or none. The logits are capped by tanh. Tensor names are the
checkpoint's: ``embed``, ``l<i>.norm1|norm2``, ``l<i>.hc1.*|hc2.*``, ``l<i>.mix.*``, ``l<i>.mlp.*``, ``final.norm``, ``head``.
"""

from __future__ import annotations

from ..config.registry import Architecture, register_architecture
from ..config.spec import LayerSpec, ModelSpec, PartSpec, RunEntry
from ..config.tunadra import TunadraConfig, TunadraLayer, complete_from_shapes


def _attention(width: int, eps: float, c) -> PartSpec:
    return PartSpec("gqa_attention", dict(
        hidden=width, heads=int(c["heads"]), kv_heads=int(c["kv_heads"]), head_dim=int(c["dim"]), value_dim=int(c["vdim"]),
        scale=float(c["scale"]), qk_norm="unit", qk_norm_eps=eps, out_gate="head_sigmoid", value_mix=bool(c.get("v_mix", False)),
        names=dict(q="q", k="k", v="v", o="o", gate="g", v_share="vmix")))


def _wkv(width: int, eps: float, c) -> PartSpec:
    return PartSpec("time_mix", dict(
        hidden=width, heads=int(c["heads"]), head_dim=int(c["dim"]), decay_rank=int(c["decay_rank"]), eps=eps,
        names=dict(r="r", k="k", v="v", g="g", o="o", norm="norm", w1="w1", w2="w2", w0="w0", u="u", mu="mu.")))


MIXERS = {"attention": _attention, "wkv": _wkv}


def _feed_forward(width: int, mlp) -> PartSpec | None:
    if mlp is None:
        return None
    r, shared = mlp["router"], mlp.get("shared")
    groups = r.get("groups") or {"count": 1, "keep": 1}
    return PartSpec("routed_experts", dict(
        hidden=width, intermediate=int(mlp["expert"]["ff"]), experts=int(r["experts"]), top=int(r["top"]), score="sigmoid",
        group_count=int(groups["count"]), group_keep=int(groups["keep"]), group_best=2, weight_scale=float(r.get("scale", 1.0)),
        renormalize=True, renorm_eps=1e-20, correction=False, activation="clamped_glu", limit=float(mlp["expert"]["limit"]),
        shared=int(shared["ff"]) if shared else 0, shared_gated=False, shared_glu=dict(limit=float(shared["limit"])) if shared else None,
        names=dict(router="router", expert="e{}.", gate="gate", up="up", down="down", shared="shared.")))


def _layer(cfg: TunadraConfig, i: int, layer: TunadraLayer, norm: PartSpec) -> LayerSpec:
    ffn = _feed_forward(cfg.width, layer.mlp)
    names = dict(mixer="mix.", norm1="norm1", links1="hc1.")
    norms = dict(norm1=norm)
    if ffn is not None:
        names.update(feed_forward="mlp.", norm2="norm2", links2="hc2.")
        norms["norm2"] = norm
    return LayerSpec(prefix=f"l{i}.", block=PartSpec("linked_streams", dict(names=names, streams=cfg.streams)),
                     mixer=MIXERS[layer.type](cfg.width, cfg.eps, layer.mixer), feed_forward=ffn, norms=norms)


def tunadra_model_spec(cfg: TunadraConfig) -> ModelSpec:
    norm = PartSpec("rmsnorm", dict(size=cfg.width, eps=cfg.eps, name=""))
    layers = tuple(_layer(cfg, i, layer, norm) for i, layer in enumerate(cfg.layers))
    # a layer without a feed-forward has nothing for its second norm and links, nor an attention layer that shares no values for a share: a
    # checkpoint may carry their tensors all the same
    spare = tuple(f"l{i}.{k}" for i, layer in enumerate(cfg.layers) if layer.mlp is None for k in ("norm2", "hc2.in", "hc2.out", "hc2.mix"))
    spare += tuple(f"l{i}.mix.vmix" for i, layer in enumerate(cfg.layers) if layer.type == "attention" and not layer.mixer.get("v_mix"))
    return ModelSpec(
        architecture="Tunadra", hidden_size=cfg.width, vocab_size=cfg.vocab,
        embedding=PartSpec("summed_embedding", dict(vocab=cfg.vocab, hidden=cfg.width, name="embed", sinusoid=10000.0, scale=cfg.embedding_scale)),
        layers=layers, run_order=tuple(RunEntry(i) for i in range(len(layers))), final_norm=norm, final_norm_prefix="final.norm",
        head=PartSpec("linear_head", dict(vocab=cfg.vocab, hidden=cfg.width, tied=False, name="head", softcap=cfg.logit_softcap)),
        optional_tensors=spare)


TUNADRA = register_architecture(Architecture("Tunadra", TunadraConfig.from_dict, tunadra_model_spec, complete_from_shapes), replace=True)
