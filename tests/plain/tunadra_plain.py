"""The Tunadra decoder restated in plain PyTorch: whole sequences, no cache, one function per mechanism.

Written from the design's equations and used as the oracle of the tests; it shares no code with the engine.
``weights`` maps tensor names to tensors; ``cfg`` is the config.json dict. ``dtype`` float32 computes everything
in 32-bit (products summed in 64-bit, so that their order does not matter); bfloat16 rounds the products' inputs and
outputs to bfloat16 where the engine may, and keeps in 32-bit what the design keeps there (norms, the router,
angles, scores, the streams and their mixing, the recurrence and what enters it)."""

from __future__ import annotations

import numpy as np
import torch


def _lin(x: torch.Tensor, w: torch.Tensor, dtype) -> torch.Tensor:
    if dtype == torch.float32:
        return (x.double() @ w.double().t()).float()
    return (x.to(dtype).float() @ w.to(dtype).float().t()).to(dtype).float()


def _r(x: torch.Tensor, dtype) -> torch.Tensor:
    return x if dtype == torch.float32 else x.to(dtype).float()


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    x = x if x.dtype == torch.float64 else x.float()
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


# ---------------------------------------------------------------------------------------------- embedding
def sinusoid(positions: torch.Tensor, width: int) -> torch.Tensor:
    """[T, width]: sin (even entries) and cos (odd ones) of position * 10000^(-2i / width), i the pair's number."""
    i = np.arange((width + 1) // 2, dtype=np.float64)
    f = torch.from_numpy((10000.0 ** (-2.0 * i / width)).astype(np.float32))
    ang = (positions.float()[:, None] * f[None, :]).double()  # a 32-bit angle
    out = torch.stack((torch.sin(ang), torch.cos(ang)), dim=-1).reshape(len(positions), -1)
    return out[:, :width].float()


def embed(cfg: dict, w: dict, tokens) -> torch.Tensor:
    scale = float(cfg["embedding"]["scale"])
    x = w["embed"].float()[torch.tensor([int(t) for t in tokens], dtype=torch.long)] * scale
    return x + sinusoid(torch.arange(len(tokens)), x.shape[1])


# ---------------------------------------------------------------------------------------------- several streams
def gather_streams(streams: torch.Tensor, into: torch.Tensor) -> torch.Tensor:
    """streams [T, S, W], into [S] -> the sublayer's input [T, W]."""
    return (streams * into.float()[None, :, None]).sum(1)


def update_streams(streams: torch.Tensor, y: torch.Tensor, mix: torch.Tensor, out: torch.Tensor) -> torch.Tensor:
    """Stream t of the result = sum over s of mix[s, t] * (old) stream s, + out[t] * y."""
    n = streams.shape[1]
    new = torch.zeros_like(streams)
    for t in range(n):
        for s in range(n):
            new[:, t] += mix.float()[s, t] * streams[:, s]
        new[:, t] += out.float()[t] * y
    return new


# ---------------------------------------------------------------------------------------------- attention
def mix_values(v: torch.Tensor, first: torch.Tensor, share: torch.Tensor) -> torch.Tensor:
    """(1 - share) v + share first, share one number."""
    return (1.0 - share.float()) * v + share.float() * first


def attention(h: torch.Tensor, w: dict, p: str, m: dict, eps: float, dtype, shared: dict | None = None) -> torch.Tensor:
    """``shared``: what layers hand on to later ones; "v" holds the first v_mix layer's values [T, kv_heads * vdim]."""
    heads, kv, dim, vd = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    t = h.shape[0]
    pos = torch.arange(t)
    q = _r(rms(_lin(h, w[p + "q"], dtype).view(t, heads, dim), eps), dtype)
    k = _r(rms(_lin(h, w[p + "k"], dtype).view(t, kv, dim), eps), dtype)
    v = _lin(h, w[p + "v"], dtype)
    if m.get("v_mix"):
        if shared is not None and "v" in shared:
            v = _r(mix_values(v, shared["v"], w[p + "vmix"]), dtype)
        elif shared is not None:
            shared["v"] = v
    v = v.view(t, kv, vd)
    gate = torch.sigmoid(_lin(h, w[p + "g"], dtype))
    out = torch.zeros(t, heads, vd)
    for hd in range(heads):
        g = hd // (heads // kv)
        s = (q[:, hd].double() @ k[:, g].double().t()).float() * float(m["scale"])
        s = s.masked_fill(pos[None, :] > pos[:, None], float("-inf"))
        out[:, hd] = (_r(torch.softmax(s, dim=-1), dtype).double() @ v[:, g].double()).float() * gate[:, hd, None]
    return _lin(_r(out.reshape(t, heads * vd), dtype), w[p + "o"], dtype)


# ---------------------------------------------------------------------------------------------- time mixing
def previous(h: torch.Tensor) -> torch.Tensor:
    """Every token's predecessor; zeros ahead of the first."""
    return torch.cat((torch.zeros_like(h[:1]), h[:-1]), dim=0)


def shift_mix(h: torch.Tensor, mu: torch.Tensor) -> torch.Tensor:
    return h + (previous(h) - h) * mu.float()[None, :]


def channel_decay(z: torch.Tensor) -> torch.Tensor:
    return torch.exp(-torch.exp(z))


def bonus_scan(r, k, v, decay, u) -> torch.Tensor:
    """r, k, decay [T, H, d], v [T, H, e], u [H, d] -> [T, H, e], token by token, as the equations stand: the read-out sees the
    state before the token's own write, and the token's own k v^T times u."""
    t, heads, d = r.shape
    s = torch.zeros(heads, d, v.shape[2], dtype=r.dtype)
    out = torch.zeros(t, heads, v.shape[2], dtype=r.dtype)
    for x in range(t):
        kv = k[x][:, :, None] * v[x][:, None, :]
        out[x] = ((s + u[:, :, None] * kv) * r[x][:, :, None]).sum(1)
        s = decay[x][:, :, None] * s + kv
    return out


def wkv(h: torch.Tensor, w: dict, p: str, m: dict, eps: float, dtype, shared: dict | None = None, acc=torch.float32) -> torch.Tensor:
    heads, dim = int(m["heads"]), int(m["dim"])
    t = h.shape[0]
    mixed = {x: _r(shift_mix(h, w[f"{p}mu.{x}"]), dtype) for x in ("r", "k", "v", "g", "w")}
    r, k, v = (_lin(mixed[x], w[p + x], dtype).view(t, heads, dim).to(acc) for x in ("r", "k", "v"))
    gate = silu(_lin(mixed["g"], w[p + "g"], dtype))
    low = _r(torch.tanh(_lin(mixed["w"], w[p + "w1"], dtype)), dtype)
    z = (low.double() @ _r(w[p + "w2"].float(), dtype).double().t()).to(acc) + w[p + "w0"].to(acc)
    o = bonus_scan(r, k, v, channel_decay(z).view(t, heads, dim), w[p + "u"].to(acc))
    o = rms(o, eps).reshape(t, heads * dim).float() * w[p + "norm"].float() * gate
    return _lin(_r(o, dtype), w[p + "o"], dtype)


# ---------------------------------------------------------------------------------------------- feed-forward
def clamped_glu(g: torch.Tensor, u: torch.Tensor, limit: float) -> torch.Tensor:
    g, u = torch.clamp(g, max=limit), torch.clamp(u, -limit, limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1.0)


def route(h: torch.Tensor, w: dict, p: str, router: dict, dtype) -> tuple[torch.Tensor, torch.Tensor]:
    """(chosen [T, top], weights [T, top])."""
    top = int(router["top"])
    s = torch.sigmoid((_r(h, dtype).double() @ w[p + "router"].double().t()).float())
    choice = s.clone()
    groups = router.get("groups")
    if groups:
        count, keep = int(groups["count"]), int(groups["keep"])
        per = s.shape[1] // count
        score = torch.sort(s.view(-1, count, per), dim=-1, descending=True).values[..., :2].sum(-1)
        kept = torch.topk(score, keep, dim=-1).indices
        allowed = torch.zeros(s.shape[0], count, dtype=torch.bool).scatter_(1, kept, True)
        choice = choice.masked_fill(~allowed.repeat_interleave(per, dim=1), float("-inf"))
    chosen = torch.topk(choice, top, dim=-1).indices
    weights = torch.gather(s, 1, chosen)
    weights = weights / (weights.sum(-1, keepdim=True) + 1e-20) * float(router.get("scale", 1.0))
    return chosen, weights


def expert(x, w, p, limit: float, dtype):
    a = clamped_glu(_lin(x, w[p + "gate"], dtype), _lin(x, w[p + "up"], dtype), limit)
    return _lin(_r(a, dtype), w[p + "down"], dtype)


def moe_ff(h, w, p, mlp: dict, dtype):
    chosen, weights = route(h, w, p, mlp["router"], dtype)
    out = torch.zeros(h.shape[0], h.shape[1])
    for e in range(int(mlp["router"]["experts"])):
        for c in range(chosen.shape[1]):
            at = torch.nonzero(chosen[:, c] == e).flatten()
            if len(at):
                out[at] += weights[at, c][:, None] * expert(h[at], w, f"{p}e{e}.", float(mlp["expert"]["limit"]), dtype)
    if mlp.get("shared"):
        out = out + expert(h, w, p + "shared.", float(mlp["shared"]["limit"]), dtype)
    return out


# ---------------------------------------------------------------------------------------------- the model
def softcap(z: torch.Tensor, cap: float) -> torch.Tensor:
    return cap * torch.tanh(z / cap)


def forward(cfg: dict, w: dict, tokens, dtype=torch.float32, layers_out: list | None = None) -> torch.Tensor:
    """Logits [T, vocab] (float32) of one sequence; ``layers_out`` receives the sum of the streams after every layer."""
    eps = float(cfg["norm"]["eps"])
    mixers = {"attention": attention, "wkv": wkv}
    x = embed(cfg, w, tokens)[:, None, :].repeat(1, int(cfg["streams"]), 1)
    shared: dict = {}
    for n, layer in enumerate(cfg["layers"]):
        p = f"l{n}."
        for q in (1, 2):
            if q == 2 and layer.get("mlp") is None:
                continue
            h = _r(rms(gather_streams(x, w[f"{p}hc{q}.in"]), eps) * w[f"{p}norm{q}"].float(), dtype)
            if q == 1:
                y = mixers[layer["type"]](h, w, p + "mix.", layer["mixer"], eps, dtype, shared)
            else:
                y = moe_ff(h, w, p + "mlp.", layer["mlp"], dtype)
            x = update_streams(x, _r(y, dtype), w[f"{p}hc{q}.mix"], w[f"{p}hc{q}.out"])
        if layers_out is not None:
            layers_out.append(x.sum(1))
    logits = _lin(_r(rms(x.sum(1), eps) * w["final.norm"].float(), dtype), w["head"], dtype)
    return softcap(logits, float(cfg["logit_softcap"]))
