"""The Vumedra decoder as data: its configuration mapped onto parts.

The stream starts as a sum of three: the token's row, a row of a bigram table (a hash of the previous token and the token; the
previous token is state of the request) and a sinusoidal vector of the position. Every layer has an RMS norm before and after
each sublayer, the norms' weights single numbers. Three mixers: ``attention`` (grouped heads with a key and a value size,
biases on q, k and v, normed queries and keys, no rotation, a temperature of the queries that grows with the position, a
sink of score 0), ``mlstm`` (a matrix memory with exponential gates and a running maximum) and ``rglru`` (a gated linear
recurrence behind a short convolution, times a GELU branch). Feed-forward: SiLU-gated and dense, or a mixture of experts
without a gate (the square of relu), chosen and weighed by sigmoid scores that multiply the experts' inputs, beside a shared
expert; or none. Tensor names are the checkpoint's: ``embed``, ``bigram``, ``l<i>.norm1|norm1b|norm2|norm2b``, ``l<i>.mix.*``,
``l<i>.mlp.*``, ``final.norm``, ``head``.
"""

from __future__ import annotations

from ..config.registry import Architecture, register_architecture
from ..config.spec import LayerSpec, ModelSpec, PartSpec, RunEntry
from ..config.vumedra import VumedraConfig, VumedraLayer


def _attention(width: int, eps: float, c) -> PartSpec:
    temp = c.get("q_temp")
    return PartSpec("gqa_attention", dict(
        hidden=width, heads=int(c["heads"]), kv_heads=int(c["kv_heads"]), head_dim=int(c["dim"]), value_dim=int(c["vdim"]),
        scale=float(c["scale"]), qk_norm=True, qk_norm_eps=eps, qkv_bias=True, sink=True, general=True,
        query_temperature=(float(temp["coef"]), float(temp["every"])) if temp else None,
        names=dict(q="q", k="k", v="v", o="o", q_norm="q.norm", k_norm="k.norm", q_bias="q.b", k_bias="k.b", v_bias="v.b")))


def _mlstm(width: int, eps: float, c) -> PartSpec:
    return PartSpec("mlstm", dict(
        hidden=width, heads=int(c["heads"]), key_dim=int(c["dim"]), value_dim=int(c["vdim"]), gate_cap=float(c["gate_cap"]), eps=eps,
        names=dict(q="q", k="k", v="v", g="g", o="o", norm="norm", i="i", f="f", i_bias="i.b", f_bias="f.b")))


def _rglru(width: int, eps: float, c) -> PartSpec:
    return PartSpec("rglru", dict(
        hidden=width, width=int(c["width"]), blocks=int(c["blocks"]), conv=int(c["conv"]),
        names=dict(y="y", y_bias="y.b", x="x", x_bias="x.b", conv="conv", conv_bias="conv.b", r="ra", r_bias="ra.b", i="ri", i_bias="ri.b",
                   lam="lam", o="o")))


MIXERS = {"attention": _attention, "mlstm": _mlstm, "rglru": _rglru}


def _feed_forward(width: int, mlp) -> PartSpec | None:
    if mlp is None:
        return None
    if mlp["kind"] == "dense":
        return PartSpec("swiglu", dict(hidden=width, intermediate=int(mlp["ff"]), names=dict(gate="gate", up="up", down="down")))
    r, shared = mlp["router"], mlp.get("shared")
    return PartSpec("routed_experts", dict(
        hidden=width, intermediate=int(mlp["expert"]["ff"]), experts=int(r["experts"]), top=int(r["top"]), score="sigmoid", renormalize=False,
        correction=False, gated=False, activation="relu_squared", weigh="input", shared=int(shared["ff"]) if shared else 0, shared_gated=False,
        names=dict(router="router", expert="e{}.", up="up", down="down", shared="shared.")))


def _layer(cfg: VumedraConfig, i: int, layer: VumedraLayer, norm: PartSpec) -> LayerSpec:
    ffn = _feed_forward(cfg.width, layer.mlp)
    names = dict(mixer="mix.", norm1="norm1", norm1b="norm1b")
    if ffn is not None:
        names.update(feed_forward="mlp.", norm2="norm2", norm2b="norm2b")
    norms = {k: norm for k in names if k.startswith("norm")}
    return LayerSpec(prefix=f"l{i}.", block=PartSpec("sandwich", dict(names=names)), mixer=MIXERS[layer.type](cfg.width, cfg.eps, layer.mixer),
                     feed_forward=ffn, norms=norms)


def vumedra_model_spec(cfg: VumedraConfig) -> ModelSpec:
    norm = PartSpec("rmsnorm", dict(size=cfg.width, eps=cfg.eps, scalar=True, name=""))
    bigram = dict(buckets=int(cfg.bigram["buckets"]), mul_prev=int(cfg.bigram["mul_prev"]), mul_cur=int(cfg.bigram["mul_cur"]),
                  name="bigram") if cfg.bigram is not None else None
    layers = tuple(_layer(cfg, i, layer, norm) for i, layer in enumerate(cfg.layers))
    # a layer without a feed-forward has nothing for its second pair of norms: a checkpoint may carry their tensors all the same
    spare = tuple(f"l{i}.{k}" for i, layer in enumerate(cfg.layers) if layer.mlp is None for k in ("norm2", "norm2b"))
    return ModelSpec(
        architecture="Vumedra", hidden_size=cfg.width, vocab_size=cfg.vocab,
        embedding=PartSpec("summed_embedding", dict(vocab=cfg.vocab, hidden=cfg.width, name="embed", bigram=bigram, sinusoid=10000.0)),
        layers=layers, run_order=tuple(RunEntry(i) for i in range(len(layers))), final_norm=norm, final_norm_prefix="final.norm",
        head=PartSpec("linear_head", dict(vocab=cfg.vocab, hidden=cfg.width, tied=False, name="head")), optional_tensors=spare)


VUMEDRA = register_architecture(Architecture("Vumedra", VumedraConfig.from_dict, vumedra_model_spec), replace=True)
