"""Helpers of the Vumedra tests: small configurations, a model folder with random weights written from the
checkpoint format alone (names and shapes are stated here, not taken from the product), and the oracle's logits.
The runner that steps the product's own model, cache manager and step function is the one of the Fekulix tests."""

from __future__ import annotations

import copy
import json
from pathlib import Path

import torch

from tests.fekulix_util import Runner, rel_err  # noqa: F401  (shared, architecture-free)
from tests.plain import vumedra_plain as plain
from tests.rofozen_util import position_errors, rounded_ok  # noqa: F401  (architecture-free)


def dense(ff=80):
    return {"ff": ff, "kind": "dense"}


def moe(ff=24, experts=6, top=2, shared=40):
    out = {"expert": {"ff": ff}, "kind": "moe", "router": {"experts": experts, "top": top}}
    if shared:
        out["shared"] = {"ff": shared}
    return out


def attention_layer(heads=6, kv_heads=2, dim=16, vdim=24, scale=0.3, coef=0.4, every=24, mlp=None):
    mixer = {"dim": dim, "heads": heads, "kv_heads": kv_heads, "scale": scale, "vdim": vdim}
    if every:
        mixer["q_temp"] = {"coef": coef, "every": every}
    return {"type": "attention", "mixer": mixer, "mlp": mlp}


def memory_layer(heads=3, dim=16, vdim=24, cap=12.0, mlp=None):
    return {"type": "mlstm", "mixer": {"dim": dim, "gate_cap": cap, "heads": heads, "vdim": vdim}, "mlp": mlp}


def recurrent_layer(width=48, blocks=3, conv=4, mlp=None):
    return {"type": "rglru", "mixer": {"blocks": blocks, "conv": conv, "width": width}, "mlp": mlp}


def config(layers, width=64, vocab=97, eps=1e-5, buckets=131, mul_prev=37, mul_cur=11):
    return {"architecture": "Vumedra", "embedding": {"bigram": {"buckets": buckets, "mul_cur": mul_cur, "mul_prev": mul_prev}},
            "layers": copy.deepcopy(layers), "norm": {"eps": eps}, "vocab": vocab, "width": width}


def config_a():
    """Every mixer and both feed-forwards; a recurrence narrower than the model; fewer buckets than pairs of tokens."""
    return config([memory_layer(mlp=dense()), attention_layer(mlp=moe()), recurrent_layer(mlp=moe(top=3, shared=0)),
                   recurrent_layer(width=80, blocks=5, conv=3, mlp=dense(72)), memory_layer(heads=1, dim=24, vdim=16, cap=3.0, mlp=moe(top=1))])


def config_b():
    """Sizes that are no multiples of 8 where the format allows: a width of 36, five heads on one key/value head, keys of
    12 and values of 20 and the other way round, a temperature that changes at every position, one bucket, a recurrence
    in one part and in parts of 7, two taps and one, one expert of one, a layer without feed-forward, attention first and last."""
    return config([
        attention_layer(heads=5, kv_heads=1, dim=12, vdim=20, scale=0.5, coef=0.1, every=1, mlp=moe(ff=20, experts=5, top=1, shared=28)),
        recurrent_layer(width=28, blocks=4, conv=2, mlp=None),
        memory_layer(heads=5, dim=12, vdim=20, cap=7.5, mlp=moe(ff=12, experts=1, top=1, shared=0)),
        recurrent_layer(width=36, blocks=1, conv=1, mlp=dense(44)),
        attention_layer(heads=4, kv_heads=4, dim=20, vdim=12, scale=0.25, every=None, mlp=dense(52)),
    ], width=36, vocab=61, eps=1e-6, buckets=1, mul_prev=0, mul_cur=1)


def config_c():
    """Larger and rounder: a width of 256, heads of 128 on the tcgen05 kernel, a memory of 64 x 96, more buckets than the
    vocabulary has pairs of, factors whose products leave 32 bits, eight experts."""
    return config([
        recurrent_layer(width=256, blocks=2, conv=4, mlp=moe(ff=64, experts=8, top=2, shared=96)),
        attention_layer(heads=4, kv_heads=2, dim=128, vdim=128, scale=0.09, coef=0.5, every=100, mlp=dense(320)),
        memory_layer(heads=4, dim=64, vdim=96, cap=20.0, mlp=dense(192)),
        attention_layer(heads=8, kv_heads=1, dim=48, vdim=64, scale=0.15, coef=-0.2, every=40, mlp=moe(ff=48, experts=8, top=4, shared=64)),
    ], width=256, vocab=576, buckets=4099, mul_prev=10_000_019, mul_cur=8_191)


def config_d():
    """No attention at all: a model without pages, whose requests hold state slots alone."""
    return config([recurrent_layer(width=40, blocks=2, conv=3, mlp=dense(48)), memory_layer(mlp=moe())], width=48, vocab=83)


def tensor_shapes(raw) -> dict[str, tuple]:
    """Names and shapes of a checkpoint of this configuration."""
    w = raw["width"]
    out = {"embed": (raw["vocab"], w), "bigram": (raw["embedding"]["bigram"]["buckets"] + 1, w), "final.norm": (), "head": (raw["vocab"], w)}
    for i, layer in enumerate(raw["layers"]):
        p, m, q = f"l{i}.", layer["mixer"], f"l{i}.mix."
        out.update({p + "norm1": (), p + "norm1b": ()})
        if layer["type"] == "attention":
            h, g, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            out.update({q + "q": (h * dk, w), q + "q.b": (h * dk,), q + "k": (g * dk, w), q + "k.b": (g * dk,), q + "v": (g * dv, w),
                        q + "v.b": (g * dv,), q + "q.norm": (dk,), q + "k.norm": (dk,), q + "o": (w, h * dv)})
        elif layer["type"] == "mlstm":
            h, dk, dv = m["heads"], m["dim"], m["vdim"]
            out.update({q + "q": (h * dk, w), q + "k": (h * dk, w), q + "v": (h * dv, w), q + "g": (h * dv, w), q + "o": (w, h * dv),
                        q + "norm": (h * dv,), q + "i": (h, w), q + "i.b": (h,), q + "f": (h, w), q + "f.b": (h,)})
        else:
            c, b = m["width"], m["blocks"]
            s = c // b
            out.update({q + "y": (c, w), q + "y.b": (c,), q + "x": (c, w), q + "x.b": (c,), q + "conv": (c, m["conv"]), q + "conv.b": (c,),
                        q + "ra": (b, s, s), q + "ra.b": (b, s), q + "ri": (b, s, s), q + "ri.b": (b, s), q + "lam": (c,), q + "o": (w, c)})
        mlp = layer["mlp"]
        if mlp is None:
            continue
        out.update({p + "norm2": (), p + "norm2b": ()})
        f = p + "mlp."
        if mlp["kind"] == "dense":
            out.update({f + "gate": (mlp["ff"], w), f + "up": (mlp["ff"], w), f + "down": (w, mlp["ff"])})
        else:
            ff = mlp["expert"]["ff"]
            out[f + "router"] = (mlp["router"]["experts"], w)
            for e in range(mlp["router"]["experts"]):
                out.update({f"{f}e{e}.up": (ff, w), f"{f}e{e}.down": (w, ff)})
            if mlp.get("shared"):
                sf = mlp["shared"]["ff"]
                out.update({f + "shared.up": (sf, w), f + "shared.down": (w, sf)})
    return out


def random_weights(raw, seed: int, sharpen: float = 2.0) -> dict[str, torch.Tensor]:
    """bfloat16 tensors: matrices about 1/sqrt(fan-in) so that activations are of size one, the query and key norms
    times ``sharpen`` so that attention is peaked, routers large enough for clear choices, decays and forget gates from slow
    to fast, every norm's number different."""
    gen = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(raw).items():
        leaf = name.rsplit(".", 1)[-1]
        parent = name.rsplit(".", 2)[-2] if name.count(".") else ""
        t = torch.randn(shape, generator=gen)
        if leaf in ("embed", "bigram"):
            pass
        elif leaf == "b":
            if parent == "f":
                t = torch.linspace(0.0, 5.0, max(shape[0], 2))[: shape[0]] + 0.2 * t  # memories from a few tokens to hundreds
            else:
                t = 0.3 * t
        elif leaf == "conv":
            t = 0.6 * t
        elif leaf == "router":
            t = t * (3.0 / shape[1] ** 0.5)
        elif leaf == "lam":
            t = torch.rand(shape, generator=gen) * 6.0 - 6.0  # decays per token from 0.99 to 0.06
        elif len(shape) >= 2:
            t = t * (1.2 / shape[-1] ** 0.5)
        else:  # norm weights, vectors and single numbers
            t = 1.0 + 0.25 * t
            if name.endswith(("q.norm", "k.norm")):
                t = t * sharpen
        out[name] = t.to(torch.bfloat16)
    return out


def write_model(folder, raw, seed: int, sharpen: float = 2.0, change=None) -> Path:
    from safetensors.torch import save_file

    folder = Path(folder)
    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(raw, indent=1))
    w = random_weights(raw, seed, sharpen)
    if change:
        change(w)
    save_file({k: v.contiguous() for k, v in w.items()}, str(folder / "model.safetensors"))
    return folder


def read_weights(folder) -> dict[str, torch.Tensor]:
    from safetensors.torch import load_file

    return {k: v.float() for k, v in load_file(str(Path(folder) / "model.safetensors")).items()}


def oracle(folder, dtype=torch.float32):
    """ids -> logits [T, vocab] of the plain implementation (32-bit: products summed in 64-bit)."""
    raw = json.loads((Path(folder) / "config.json").read_text())
    w = read_weights(folder)
    return lambda ids: plain.forward(raw, w, ids, dtype)


def float32_ok(folder, got: torch.Tensor, want: torch.Tensor, ids, limit: float) -> tuple[bool, str]:
    """Whether 32-bit logits are within ``limit`` of the oracle's at every position (distance over the spread). A memory's read-out
    is divided by its own size and normed: where a query is nearly orthogonal to all that a head holds (the first token with
    k . q near zero), 32-bit rounding itself shows. So a position beyond the limit is compared with how far the oracle moves
    when every weight is moved by one part in ten million, and may be four times as far."""
    err = position_errors(got, want)
    if err.max() < limit:
        return True, ""
    raw = json.loads((Path(folder) / "config.json").read_text())
    w = read_weights(folder)
    moved = torch.zeros_like(err)
    for seed in range(3):
        gen = torch.Generator().manual_seed(seed)
        near = {k: v * (1.0 + 1e-7 * torch.randn(v.shape, generator=gen)) for k, v in w.items()}
        moved = torch.maximum(moved, position_errors(plain.forward(raw, near, ids), want))
    bad = err > torch.clamp(4.0 * moved, min=limit)
    at = int(err.argmax())
    return not bad.any(), f"{int(bad.sum())} positions off, the worst {err[at]:.2e} at {at} (rounding alone: {moved[at]:.2e})"


def layer_streams(folder, ids) -> list[torch.Tensor]:
    raw = json.loads((Path(folder) / "config.json").read_text())
    out: list = []
    plain.forward(raw, read_weights(folder), ids, torch.float32, out)
    return out
