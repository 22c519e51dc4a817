"""The Vumedra decoder restated in plain PyTorch: whole sequences, no cache, one function per mechanism.

Written from the design's equations and used as the oracle of the tests; it shares no code with the engine.
``weights`` maps tensor names to tensors; ``cfg`` is the config.json dict. ``dtype`` float32 computes everything
in 32-bit (products summed in 64-bit, so that their order does not matter); bfloat16 rounds the products' inputs and
outputs to bfloat16 where the engine may, and keeps in 32-bit what the design keeps there (norms, routers, angles,
scores, the residual sum, the recurrences and what enters them)."""

from __future__ import annotations

import math

import numpy as np
import torch


def _lin(x: torch.Tensor, w: torch.Tensor, dtype) -> torch.Tensor:
    if dtype == torch.float32:
        return (x.double() @ w.double().t()).float()
    return (x.to(dtype).float() @ w.to(dtype).float().t()).to(dtype).float()


def _r(x: torch.Tensor, dtype) -> torch.Tensor:
    return x if dtype == torch.float32 else x.to(dtype).float()


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    x = x.float()
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def scalar_norm(x: torch.Tensor, g: torch.Tensor, eps: float) -> torch.Tensor:
    """An RMS norm whose scale is one number for all coordinates."""
    return rms(x, eps) * g.float().reshape(())


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z * torch.sigmoid(z)


def relu_squared(z):
    return torch.relu(z) ** 2


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


# ---------------------------------------------------------------------------------------------- embedding
def bigram_rows(tokens, buckets: int, mul_prev: int, mul_cur: int) -> torch.Tensor:
    """Row of the bigram table at every position: a hash of (previous token, token); the first token has a row of its own."""
    rows = [buckets]
    for prev, cur in zip(tokens[:-1], tokens[1:]):
        rows.append((int(prev) * mul_prev + int(cur) * mul_cur) % buckets)
    return torch.tensor(rows[: len(tokens)], dtype=torch.long)


def sinusoid(positions: torch.Tensor, width: int) -> torch.Tensor:
    """[T, width]: sin (even entries) and cos (odd ones) of position * 10000^(-2i / width), i the pair's number."""
    i = np.arange((width + 1) // 2, dtype=np.float64)
    f = torch.from_numpy((10000.0 ** (-2.0 * i / width)).astype(np.float32))
    ang = (positions.float()[:, None] * f[None, :]).double()  # a 32-bit angle
    out = torch.stack((torch.sin(ang), torch.cos(ang)), dim=-1).reshape(len(positions), -1)
    return out[:, :width].float()


def embed(cfg: dict, w: dict, tokens) -> torch.Tensor:
    tokens = [int(t) for t in tokens]
    b = cfg["embedding"]["bigram"]
    x = w["embed"].float()[torch.tensor(tokens, dtype=torch.long)]
    x = x + w["bigram"].float()[bigram_rows(tokens, int(b["buckets"]), int(b["mul_prev"]), int(b["mul_cur"]))]
    return x + sinusoid(torch.arange(len(tokens)), x.shape[1])


# ---------------------------------------------------------------------------------------------- attention
def query_temperature(positions: torch.Tensor, coef: float, every: float) -> torch.Tensor:
    return 1.0 + coef * torch.log(torch.floor((positions.float() + 1.0) / every) + 1.0)


def sink_softmax(scores: torch.Tensor) -> torch.Tensor:
    """exp(s) over 1 + the sum of exp(s): one more term of score 0 in the denominator."""
    m = torch.clamp(scores.max(dim=-1, keepdim=True).values, min=0.0)
    e = torch.exp(scores - m)
    return e / (torch.exp(-m) + e.sum(-1, keepdim=True))


def attention(h: torch.Tensor, w: dict, p: str, m: dict, eps: float, dtype) -> torch.Tensor:
    heads, kv, dim, vd = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    t = h.shape[0]
    pos = torch.arange(t)
    q = (_lin(h, w[p + "q"], dtype) + w[p + "q.b"].float()).view(t, heads, dim)
    k = (_lin(h, w[p + "k"], dtype) + w[p + "k.b"].float()).view(t, kv, dim)
    v = _r(_lin(h, w[p + "v"], dtype) + w[p + "v.b"].float(), dtype).view(t, kv, vd)
    q = rms(q, eps) * w[p + "q.norm"].float()
    k = _r(rms(k, eps) * w[p + "k.norm"].float(), dtype)
    temp = m.get("q_temp")
    if temp:
        q = q * query_temperature(pos, float(temp["coef"]), float(temp["every"]))[:, None, None]
    q = _r(q, dtype)
    out = torch.zeros(t, heads, vd)
    for hd in range(heads):
        g = hd // (heads // kv)
        s = (q[:, hd].double() @ k[:, g].double().t()).float() * float(m["scale"])
        s = s.masked_fill(pos[None, :] > pos[:, None], float("-inf"))
        out[:, hd] = (_r(sink_softmax(s), dtype).double() @ v[:, g].double()).float()
    return _lin(_r(out.reshape(t, heads * vd), dtype), w[p + "o"], dtype)


# ---------------------------------------------------------------------------------------------- matrix memory
def mlstm_gates(i_raw: torch.Tensor, f_raw: torch.Tensor, cap: float) -> tuple[torch.Tensor, torch.Tensor]:
    """(log input gate, log forget gate) from the gates' pre-activations (biases included)."""
    return cap * torch.tanh(i_raw / cap), -softplus(-cap * torch.tanh(f_raw / cap))


def mlstm_memory(q, k, v, log_i, log_f) -> torch.Tensor:
    """q, k [T, H, dk], v [T, H, dv], gates [T, H] -> [T, H, dv], token by token, as the equations stand."""
    t, heads, dk = q.shape
    dv = v.shape[2]
    s = torch.zeros(heads, dk, dv, dtype=q.dtype)
    n = torch.zeros(heads, dk, dtype=q.dtype)
    m = torch.zeros(heads, dtype=q.dtype)
    out = torch.zeros(t, heads, dv, dtype=q.dtype)
    for x in range(t):
        new = torch.maximum(log_f[x] + m, log_i[x])
        a, b = torch.exp(log_f[x] + m - new), torch.exp(log_i[x] - new)
        s = a[:, None, None] * s + b[:, None, None] * (k[x][:, :, None] * v[x][:, None, :])
        n = a[:, None] * n + b[:, None] * k[x]
        m = new
        den = torch.maximum((n * q[x]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out[x] = (s * q[x][:, :, None]).sum(1) / den[:, None]
    return out


def mlstm(h: torch.Tensor, w: dict, p: str, m: dict, eps: float, dtype, acc=torch.float32) -> torch.Tensor:
    heads, dk, dv, cap = int(m["heads"]), int(m["dim"]), int(m["vdim"]), float(m["gate_cap"])
    t = h.shape[0]
    q = _lin(h, w[p + "q"], dtype).view(t, heads, dk).to(acc) * dk ** -0.5
    k = _lin(h, w[p + "k"], dtype).view(t, heads, dk).to(acc)
    v = _lin(h, w[p + "v"], dtype).view(t, heads, dv).to(acc)
    log_i, log_f = mlstm_gates(_lin(h, w[p + "i"], dtype).to(acc) + w[p + "i.b"].to(acc), _lin(h, w[p + "f"], dtype).to(acc) + w[p + "f.b"].to(acc), cap)
    o = mlstm_memory(q, k, v, log_i, log_f)
    o = (o / torch.sqrt((o * o).mean(-1, keepdim=True) + eps)).reshape(t, heads * dv).float() * w[p + "norm"].float()
    o = o * torch.sigmoid(_lin(h, w[p + "g"], dtype))
    return _lin(_r(o, dtype), w[p + "o"], dtype)


# ---------------------------------------------------------------------------------------------- gated linear recurrence
def causal_conv(x: torch.Tensor, w: torch.Tensor, b: torch.Tensor) -> torch.Tensor:
    """x [T, C]; w [C, taps], the last column is the current token's; zeros before the start."""
    t, c = x.shape
    taps = w.shape[1]
    pad = torch.cat((torch.zeros(taps - 1, c), x.float()), dim=0)
    out = b.float()[None, :].repeat(t, 1)
    for j in range(taps):
        out = out + pad[j: j + t] * w.float()[:, j][None, :]
    return out


def block_linear(u: torch.Tensor, w: torch.Tensor, b: torch.Tensor) -> torch.Tensor:
    """u [T, W] in as many equal parts as w [blocks, out, in] has blocks, each times its own matrix; b [blocks, out]."""
    t = u.shape[0]
    blocks = w.shape[0]
    z = torch.einsum("tbi,boi->tbo", u.view(t, blocks, -1).double(), w.double()).float() + b.float()[None]
    return z.reshape(t, -1)


def rglru_scan(u: torch.Tensor, r: torch.Tensor, i: torch.Tensor, lam: torch.Tensor) -> torch.Tensor:
    """S_t = a_t S_(t-1) + sqrt(1 - a_t^2) i_t u_t with log a_t = -8 r_t softplus(lam), from zero."""
    log_a = -8.0 * r * softplus(lam)[None, :]
    a = torch.exp(log_a)
    b = torch.sqrt(-torch.expm1(2.0 * log_a)) * i * u
    s = torch.zeros(u.shape[1], dtype=u.dtype)
    out = torch.zeros_like(u)
    for t in range(u.shape[0]):
        s = a[t] * s + b[t]
        out[t] = s
    return out


def rglru(h: torch.Tensor, w: dict, p: str, m: dict, eps: float, dtype) -> torch.Tensor:
    y = gelu_tanh(_lin(h, w[p + "y"], dtype) + w[p + "y.b"].float())
    u = _r(causal_conv(_lin(h, w[p + "x"], dtype) + w[p + "x.b"].float(), w[p + "conv"], w[p + "conv.b"]), dtype)
    r = torch.sigmoid(block_linear(u, w[p + "ra"], w[p + "ra.b"]))
    i = torch.sigmoid(block_linear(u, w[p + "ri"], w[p + "ri.b"]))
    s = rglru_scan(u, r, i, w[p + "lam"].float())
    return _lin(_r(s * y, dtype), w[p + "o"], dtype)


# ---------------------------------------------------------------------------------------------- feed-forward
def dense_ff(h, w, p, dtype):
    a = silu(_lin(h, w[p + "gate"], dtype)) * _lin(h, w[p + "up"], dtype)
    return _lin(_r(a, dtype), w[p + "down"], dtype)


def route(h: torch.Tensor, w: dict, p: str, top: int, dtype) -> tuple[torch.Tensor, torch.Tensor]:
    """(chosen [T, top], weights [T, top]): the largest sigmoid scores, as they are."""
    z = (_r(h, dtype).double() @ w[p + "router"].double().t()).float()
    s = torch.sigmoid(z)
    chosen = torch.topk(s, top, dim=-1).indices
    return chosen, torch.gather(s, 1, chosen)


def expert(x, w, p, dtype):
    return _lin(_r(relu_squared(_lin(x, w[p + "up"], dtype)), dtype), w[p + "down"], dtype)


def moe_ff(h, w, p, mlp: dict, dtype):
    chosen, weights = route(h, w, p, int(mlp["router"]["top"]), dtype)
    out = torch.zeros(h.shape[0], h.shape[1])
    for e in range(int(mlp["router"]["experts"])):
        for c in range(chosen.shape[1]):
            at = torch.nonzero(chosen[:, c] == e).flatten()
            if len(at):
                out[at] += expert(weights[at, c][:, None] * h[at], w, f"{p}e{e}.", dtype)
    if mlp.get("shared"):
        out = out + expert(h, w, p + "shared.", dtype)
    return out


# ---------------------------------------------------------------------------------------------- the model
def forward(cfg: dict, w: dict, tokens, dtype=torch.float32, layers_out: list | None = None) -> torch.Tensor:
    """Logits [T, vocab] (float32) of one sequence; ``layers_out`` receives the stream after every layer."""
    eps = float(cfg["norm"]["eps"])
    mixers = {"attention": attention, "mlstm": mlstm, "rglru": rglru}
    x = embed(cfg, w, tokens)
    for n, layer in enumerate(cfg["layers"]):
        p = f"l{n}."
        h = _r(scalar_norm(x, w[p + "norm1"], eps), dtype)
        x = x + scalar_norm(_r(mixers[layer["type"]](h, w, p + "mix.", layer["mixer"], eps, dtype), dtype), w[p + "norm1b"], eps)
        mlp = layer.get("mlp")
        if mlp is not None:
            h = _r(scalar_norm(x, w[p + "norm2"], eps), dtype)
            y = dense_ff(h, w, p + "mlp.", dtype) if mlp["kind"] == "dense" else moe_ff(h, w, p + "mlp.", mlp, dtype)
            x = x + scalar_norm(_r(y, dtype), w[p + "norm2b"], eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    return _lin(_r(scalar_norm(x, w["final.norm"], eps), dtype), w["head"], dtype)
