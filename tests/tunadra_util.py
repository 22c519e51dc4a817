"""Helpers of the Tunadra tests: small configurations, a model folder with random weights written from the
checkpoint format alone (names and shapes are stated here, not taken from the product), and the oracle's logits.
The runner that steps the product's own model, cache manager and step function is the one of the Fekulix tests."""

from __future__ import annotations

import copy
import json
from pathlib import Path

import torch

from tests.fekulix_util import Runner, rel_err  # noqa: F401  (shared, architecture-free)
from tests.plain import tunadra_plain as plain
from tests.rofozen_util import position_errors, rounded_ok  # noqa: F401  (architecture-free)


def moe(ff=24, experts=6, top=2, count=3, keep=2, scale=1.7, limit=1.5, shared=40, shared_limit=0.8):
    out = {"expert": {"ff": ff, "limit": limit}, "kind": "moe", "router": {"experts": experts, "scale": scale, "top": top}}
    if count:
        out["router"]["groups"] = {"count": count, "keep": keep}
    if shared:
        out["shared"] = {"ff": shared, "limit": shared_limit}
    return out


def attention_layer(heads=6, kv_heads=2, dim=16, vdim=24, scale=0.3, v_mix=True, mlp=None):
    return {"type": "attention", "mixer": {"dim": dim, "heads": heads, "kv_heads": kv_heads, "scale": scale, "v_mix": v_mix, "vdim": vdim}, "mlp": mlp}


def wkv_layer(heads=3, dim=16, rank=12, mlp=None):
    """``rank`` is not part of config.json: it is the first size of the tensor w1."""
    return {"type": "wkv", "mixer": {"dim": dim, "heads": heads}, "mlp": mlp, "rank": rank}


def config(layers, width=64, vocab=97, eps=1e-5, streams=2, scale=3.5, softcap=11.0):
    return {"architecture": "Tunadra", "embedding": {"scale": scale}, "layers": copy.deepcopy(layers), "logit_softcap": softcap,
            "norm": {"eps": eps}, "streams": streams, "vocab": vocab, "width": width}


def config_a():
    """Three streams; both mixers, heads narrower and wider than the model; values shared between two attention layers that split them
    into heads differently, with one in between that shares none; a layer without feed-forward."""
    return config([
        wkv_layer(mlp=moe()), attention_layer(mlp=moe(top=3)), attention_layer(heads=4, kv_heads=4, dim=20, vdim=12, v_mix=False, mlp=None),
        wkv_layer(heads=5, dim=24, rank=7, mlp=moe(experts=8, count=4, keep=3, top=4, shared=0)),
        attention_layer(heads=6, kv_heads=3, dim=32, vdim=16, scale=0.2, mlp=moe(experts=4, count=2, keep=1, top=2, limit=0.5))], streams=3)


def config_b():
    """Sizes that are no multiples of 8: a width of 36, heads of 6 and 10 channels, a rank of 5; one stream; one expert, experts without
    groups and groups of one expert; a single attention layer whose value flag has nothing to mix with; attention last."""
    return config([
        wkv_layer(heads=3, dim=10, rank=5, mlp=moe(ff=20, experts=5, top=1, count=0, shared=28)),
        wkv_layer(heads=1, dim=6, rank=1, mlp=moe(ff=12, experts=1, top=1, count=0, scale=0.5, shared=0)),
        wkv_layer(heads=2, dim=20, rank=16, mlp=None),
        attention_layer(heads=5, kv_heads=1, dim=12, vdim=20, scale=0.5, mlp=moe(ff=20, experts=4, count=4, keep=3, top=3, shared=12)),
    ], width=36, vocab=61, eps=1e-6, streams=1, scale=0.7, softcap=4.0)


def config_c():
    """Larger and rounder: heads of 128 on the tcgen05 kernel, time mixing in heads of 64 and 128, eight experts in two groups."""
    return config([
        wkv_layer(heads=3, dim=64, rank=32, mlp=moe(ff=64, experts=8, count=2, keep=1, top=3, shared=96)),
        attention_layer(heads=4, kv_heads=2, dim=128, vdim=128, scale=0.09, mlp=moe(ff=72, experts=8, count=4, keep=2, top=2, shared=64)),
        wkv_layer(heads=2, dim=128, rank=24, mlp=moe(ff=64, experts=8, count=2, keep=2, top=4, shared=0)),
        attention_layer(heads=8, kv_heads=4, dim=48, vdim=64, scale=0.15, mlp=moe(ff=48, experts=8, count=4, keep=3, top=4, shared=64)),
        attention_layer(heads=4, kv_heads=1, dim=64, vdim=32, scale=0.12, v_mix=False, mlp=None),
    ], width=192, vocab=530, streams=4, scale=9.0, softcap=20.0)


def config_d():
    """No attention at all: a model without pages, whose requests hold state slots alone; five streams."""
    return config([wkv_layer(heads=2, dim=32, rank=8, mlp=moe()), wkv_layer(heads=4, dim=8, rank=3, mlp=moe(shared=0))], width=48, vocab=83, streams=5)


def stored(raw) -> dict:
    """config.json as a checkpoint has it (the ranks are the tensors' sizes alone)."""
    out = copy.deepcopy(raw)
    for layer in out["layers"]:
        layer.pop("rank", None)
    return out


def resolved(raw) -> dict:
    """The configuration with the ranks filled in (what the registry makes of it with a checkpoint at hand)."""
    out = copy.deepcopy(raw)
    for layer in out["layers"]:
        rank = layer.pop("rank", None)
        if rank is not None:
            layer["mixer"]["decay_rank"] = rank
    return out


def tensor_shapes(raw) -> dict[str, tuple]:
    """Names and shapes of a checkpoint of this configuration."""
    w, st = raw["width"], raw["streams"]
    out = {"embed": (raw["vocab"], w), "final.norm": (w,), "head": (raw["vocab"], w)}
    for i, layer in enumerate(raw["layers"]):
        p, m, q, mlp = f"l{i}.", layer["mixer"], f"l{i}.mix.", layer["mlp"]
        for n in (1, 2) if mlp is not None else (1,):
            out.update({f"{p}norm{n}": (w,), f"{p}hc{n}.in": (st,), f"{p}hc{n}.out": (st,), f"{p}hc{n}.mix": (st, st)})
        if layer["type"] == "attention":
            h, g, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            out.update({q + "q": (h * dk, w), q + "k": (g * dk, w), q + "v": (g * dv, w), q + "g": (h, w), q + "o": (w, h * dv)})
            if m["v_mix"]:
                out[q + "vmix"] = ()
        else:
            c, rank = m["heads"] * m["dim"], layer["rank"]
            out.update({q + "mu." + x: (w,) for x in "rkvgw"})
            out.update({q + x: (c, w) for x in "rkvg"})
            out.update({q + "w1": (rank, w), q + "w2": (c, rank), q + "w0": (c,), q + "u": (m["heads"], m["dim"]), q + "norm": (c,), q + "o": (w, c)})
        if mlp is None:
            continue
        f, ff = p + "mlp.", mlp["expert"]["ff"]
        out[f + "router"] = (mlp["router"]["experts"], w)
        for e in range(mlp["router"]["experts"]):
            out.update({f"{f}e{e}.gate": (ff, w), f"{f}e{e}.up": (ff, w), f"{f}e{e}.down": (w, ff)})
        if mlp.get("shared"):
            sf = mlp["shared"]["ff"]
            out.update({f + "shared.gate": (sf, w), f + "shared.up": (sf, w), f + "shared.down": (w, sf)})
    return out


def random_weights(raw, seed: int) -> dict[str, torch.Tensor]:
    """bfloat16 tensors: matrices about 1/sqrt(fan-in) so that activations are of size one, routers large enough for clear choices, decays
    from one token to hundreds, streams that differ in what they give, take and pass on."""
    gen = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(raw).items():
        leaf = name.rsplit(".", 1)[-1]
        t = torch.randn(shape, generator=gen)
        if leaf == "embed":
            t = 0.5 * t
        elif ".hc" in name and leaf == "mix":
            t = 0.9 * torch.eye(shape[0]) + 0.2 * t / shape[0] ** 0.5
        elif ".hc" in name:
            t = (0.6 if leaf == "in" else 1.0) + 0.3 * t
        elif ".mu." in name:
            t = torch.rand(shape, generator=gen) * 1.4 - 0.2
        elif leaf == "w0":
            t = torch.linspace(-5.5, 1.5, shape[0])[torch.randperm(shape[0], generator=gen)]
        elif leaf == "u":
            t = 0.8 * t
        elif leaf == "vmix":
            t = 0.4 + 0.2 * t
        elif leaf == "router":
            t = t * (3.0 / shape[1] ** 0.5)
        elif leaf in ("q", "k"):
            t = t * (2.0 / shape[-1] ** 0.5)
        elif len(shape) >= 2:
            t = t * (1.2 / shape[-1] ** 0.5)
        else:
            t = 1.0 + 0.25 * t
        out[name] = t.to(torch.bfloat16)
    return out


def write_model(folder, raw, seed: int, change=None) -> Path:
    from safetensors.torch import save_file

    folder = Path(folder)
    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(stored(raw), indent=1))
    w = random_weights(raw, seed)
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
    """Whether 32-bit logits are within ``limit`` of the oracle's at every position (distance over the spread). Heads and sums of streams
    are divided by their own size, and a router may stand on an edge: where 32-bit rounding itself shows, a position is compared with how far the
    oracle moves when every weight is moved by one part in ten million, and may be four times as far."""
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
