"""Vumedra on the GPU against the plain implementation: each mechanism alone, whole prompts against
token-by-token decoding and portions down to two tokens, unequal requests in one batch against each
alone, pages and state slots that are given back and used again, keys far away and at page borders (in
prompts and in decoding), the first tokens of a sequence, long decoding, sizes that are no round numbers,
the trace runner and greedy generation through the entry point."""

import math
import random

import pytest
import torch

from miniserve_b200.cache.manager import KVEntryView, StateEntryView
from miniserve_b200.config import PartSpec
from miniserve_b200.parts import BuildEnv, ResidualStream, build_part
from tests import vumedra_util as vx
from tests.kernel_util import PagedBatch, make_context
from tests.plain import vumedra_plain as plain

pytestmark = pytest.mark.gpu
DEV = torch.device("cuda")
F32 = 1e-4  # logits in 32-bit: distance over their spread (rel_err); the oracle sums its products in 64-bit, the engine in 32-bit
DTYPES = [torch.float32, torch.bfloat16]
HIDDEN = 48


def _ids(n, vocab, seed):
    rng = random.Random(seed)
    return [rng.randrange(vocab) for _ in range(n)]


def _close(got, want, dtype, scale=1.0, noise=None):
    """``noise`` [T]: what rounding alone costs the plain form at each token (its distance from itself computed one
    precision higher); a token may be four times that far on top of the tolerance."""
    got, want = got.double().cpu(), want.double()
    tol = 2e-5 if dtype == torch.float32 else 3e-2
    err = (got - want).abs()
    allowed = torch.full((want.shape[0],), tol * scale * max(1.0, want.abs().max().item()), dtype=torch.float64)
    if noise is not None:
        allowed = allowed + 4.0 * noise.double()
    worst = err.amax(dim=tuple(range(1, err.dim())))
    bad = (~(worst <= allowed)).nonzero().flatten().tolist()
    assert not bad, f"off by {err.max().item():.3e} (values up to {want.abs().max().item():.2f}); tokens {bad[:8]}"


def _bind(part, dtype, seed=0, std=0.3, change=None):
    """Random bfloat16-exact weights bound to the part; returns them as float32 on the CPU by name."""
    gen = torch.Generator().manual_seed(seed)
    tensors = {}
    for name, decl in part.all_weights().items():
        t = torch.randn(decl.shape, generator=gen) * std
        if decl.init == "ones_normal":
            t = 1.0 + t / 2
        tensors[name] = t.to(torch.bfloat16).float()
    if change:
        change(tensors)
    tensors = {k: v.to(torch.bfloat16).float() for k, v in tensors.items()}
    part.bind_all({k: v.to(device=DEV, dtype=torch.float32 if part.all_weights()[k].precision == "float32" else dtype)
                   for k, v in tensors.items()})
    return tensors


@pytest.fixture(autouse=True)
def _seeded():
    torch.manual_seed(1357)
    torch.cuda.manual_seed(1357)


def _ctx(rows, page=8, kv_heads=1, d=16, dtype=torch.float32, slots=None, share=None, seed=0, ids=None):
    pb = PagedBatch(rows, page, kv_heads, d, dtype, seed=seed, share=share)
    ctx = make_context(pb)
    ctx.state_slot = torch.tensor(slots if slots is not None else list(range(len(rows))), dtype=torch.int32, device=DEV)
    if ids is not None:
        ctx.token_ids = torch.tensor(ids, dtype=torch.int32, device=DEV)
    return pb, ctx


def _x(n, dtype, std=1.0):
    return (torch.randn(n, HIDDEN, device=DEV) * std).to(dtype)


def _cpu(x):
    return x.float().cpu()


def _state_views(part):
    """Slots that hold rubbish (NaN, or a large integer): nothing of it may show in a sequence that starts there."""
    need = part.cache_need()
    needs = need if isinstance(need, tuple) else (need,)
    fill = {torch.int32: 123456789}
    views = tuple(StateEntryView(torch.full((5, *nd.shape), fill.get(nd.dtype, float("nan")), dtype=nd.dtype, device=DEV), tuple(nd.shape))
                  for nd in needs)
    return views if isinstance(need, tuple) else views[0]


def _state_portions(part, views, x, cuts, slot, dtype):
    outs, at = [], 0
    for size in cuts:
        size = min(size, x.shape[0] - at)
        if size <= 0:
            break
        _, ctx = _ctx([(at, size)], dtype=dtype, slots=[slot])
        outs.append(part.forward(x[at:at + size].contiguous(), ctx, views).clone())
        at += size
    return torch.cat(outs)


# --------------------------------------------------------------------------- embedding
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width, vocab, buckets, mul_prev, mul_cur", [
    (64, 97, 131, 37, 11), (45, 61, 1, 0, 1), (36, 50, 7, 5, 3), (1024, 30, 4099, 3, 1), (24, 40000, 97, 2_000_003, 65_537)])
def test_summed_embedding(dtype, width, vocab, buckets, mul_prev, mul_cur):
    emb = build_part("embedding", PartSpec("summed_embedding", dict(
        vocab=vocab, hidden=width, name="embed", sinusoid=10000.0,
        bigram=dict(buckets=buckets, mul_prev=mul_prev, mul_cur=mul_cur, name="bigram"))), BuildEnv(dtype, DEV))
    w = _bind(emb, dtype, std=1.0)
    raw = vx.config([], width=width, vocab=vocab, buckets=buckets, mul_prev=mul_prev, mul_cur=mul_cur)
    a, b = _ids(70, vocab, 1), _ids(33, vocab, 2)
    a[5:8] = [vocab - 1, vocab - 1, 0]
    want_a, want_b = plain.embed(raw, w, a), plain.embed(raw, w, b)

    def run(rows, slots, view):
        """rows: (ids, start, count)"""
        _, ctx = _ctx([(s, n) for _, s, n in rows], dtype=dtype, slots=slots, ids=[t for seq, s, n in rows for t in seq[s:s + n]])
        return emb.forward(ctx, view)

    view = _state_views(emb)
    _close(run([(a, 0, 70)], [2], view), want_a, torch.float32)
    at, outs = 0, []  # the same slot again, in portions down to one token from the first on
    for n in (1, 1, 2, 17, 2, 1, 9) + (1,) * 70:
        n = min(n, 70 - at)
        if n:
            outs.append(run([(a, at, n)], [2], view))
        at += n
    _close(torch.cat(outs), want_a, torch.float32)
    # two requests beside each other, other slots, one decoding beside a portion
    both = run([(a, 0, 20), (b, 0, 32)], [4, 0], view)
    _close(both, torch.cat((want_a[:20], want_b[:32])), torch.float32)
    both = run([(b, 32, 1), (a, 20, 31)], [0, 4], view)
    _close(both, torch.cat((want_b[32:], want_a[20:51])), torch.float32)


def test_the_first_token_has_a_bigram_row_of_its_own_and_no_other_token_has():
    emb = build_part("embedding", PartSpec("summed_embedding", dict(
        vocab=5, hidden=8, name="embed", sinusoid=None, bigram=dict(buckets=3, mul_prev=1, mul_cur=1, name="bigram"))), BuildEnv(torch.float32, DEV))
    w = _bind(emb, torch.float32, change=lambda t: (t["embed"].zero_(), t["bigram"].copy_(torch.arange(4.0)[:, None].expand(4, 8))))
    assert w["bigram"][3, 0] == 3
    view = _state_views(emb)
    for ids, start, want in (([1, 2, 2, 0], 0, [3, 0, 1, 2]), ([4], 4, [1]), ([0], 0, [3]), ([0], 1, [0])):
        _, ctx = _ctx([(start, len(ids))], slots=[1], ids=ids)
        assert emb.forward(ctx, view)[:, 0].tolist() == want


def test_sinusoid_at_far_positions():
    emb = build_part("embedding", PartSpec("summed_embedding", dict(vocab=3, hidden=64, name="embed", sinusoid=10000.0)), BuildEnv(torch.float32, DEV))
    _bind(emb, torch.float32, change=lambda t: t["embed"].zero_())
    for start in (0, 1000, 30000):
        _, ctx = _ctx([(start, 40)], ids=[0] * 40)
        _close(emb.forward(ctx), plain.sinusoid(torch.arange(start, start + 40), 64), torch.float32)


# --------------------------------------------------------------------------- norms
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [36, 45, 64, 1024, 2056, 4104, 9001])
@pytest.mark.parametrize("scalar, delta_scalar", [(True, True), (False, True), (True, False), (True, None)])
def test_norm_of_the_stream_with_a_normed_addend(dtype, width, scalar, delta_scalar):
    """One number or a vector as either norm's weight, no norm on the addend, no addend, and a gather of rows."""
    norm = build_part("norm", PartSpec("rmsnorm", dict(size=width, eps=1e-5, scalar=scalar, name="g")), BuildEnv(dtype, DEV))
    w = _bind(norm, dtype)
    inner, wb = None, None
    if delta_scalar is not None:
        inner = build_part("norm", PartSpec("rmsnorm", dict(size=width, eps=3e-4, scalar=delta_scalar, name="g")), BuildEnv(dtype, DEV))
        wb = _bind(inner, dtype, seed=5)
    n = 7
    res = torch.randn(n, width, device=DEV) * 3 + 0.5
    delta = (torch.randn(n, width, device=DEV) * torch.logspace(-3, 1, n, device=DEV)[:, None]).to(dtype)  # from far below eps to large
    d = _cpu(delta)
    h = _cpu(res) + (plain.rms(d, 3e-4) * wb["g"] if inner is not None else d)
    want = plain.rms(h, 1e-5) * w["g"]
    _, ctx = _ctx([(0, n)], dtype=dtype)
    held = res.clone()
    _close(norm.forward(held, delta, ctx, delta_norm=inner), want, dtype)
    _close(held, h, torch.float32)  # the sum goes back to the stream in 32-bit
    rows = torch.tensor([4, 0, 6], dtype=torch.int32, device=DEV)
    held = res.clone()
    _close(norm.forward(held, delta, ctx, rows=rows, num_rows=3, write_residual=False, delta_norm=inner), want[[4, 0, 6]], dtype)
    assert torch.equal(held, res)
    _close(norm.forward(res.clone(), None, ctx), plain.rms(_cpu(res), 1e-5) * w["g"], dtype)


# --------------------------------------------------------------------------- attention
def _attention(dtype, heads, kv, dim, vdim, scale=0.3, coef=0.4, every=16):
    from miniserve_b200.models.vumedra import _attention as spec_of

    m = vx.attention_layer(heads, kv, dim, vdim, scale, coef, every)["mixer"]
    return build_part("mixer", spec_of(HIDDEN, 1e-5, m), BuildEnv(dtype, DEV)), m


def _attention_ref(x, w, m):
    return plain.attention(_cpu(x), w, "", m, 1e-5, torch.float32)


def _kv_portions(part, x, cuts, page, dtype, full):
    view = KVEntryView(0, full.k_pool, full.v_pool, page)
    outs, at = [], 0
    for size in cuts:
        size = min(size, x.shape[0] - at)
        if size <= 0:
            break
        _, ctx = _ctx([(at, size)], page, part.kv_heads, part.cache_dim, dtype, share=full)
        outs.append(part.forward(x[at:at + size].contiguous(), ctx, view).clone())
        at += size
    return torch.cat(outs)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, kv, dim, vdim, page, every", [
    (6, 2, 16, 24, 16, 24), (5, 1, 12, 20, 8, 1), (4, 4, 20, 12, 8, None), (4, 2, 128, 128, 16, 10), (8, 1, 96, 64, 16, 7), (2, 1, 64, 128, 4, 33),
    (1, 1, 8, 8, 16, 2), (2, 1, 300, 40, 16, 5), (16, 2, 48, 48, 32, 12)])
def test_attention_whole_in_portions_and_decoded(dtype, heads, kv, dim, vdim, page, every):
    att, m = _attention(dtype, heads, kv, dim, vdim, scale=dim ** -0.5, every=every)
    w = _bind(att, dtype, change=lambda t: (t["q.norm"].mul_(2.0), t["q.b"].mul_(3.0), t["k.b"].mul_(3.0), t["v.b"].mul_(3.0)))
    n = 61
    x = _x(n, dtype)
    ref = _attention_ref(x, w, m)
    full, ctx = _ctx([(0, n)], page, kv, att.cache_dim, dtype, seed=1)
    out = att.forward(x, ctx, KVEntryView(0, full.k_pool, full.v_pool, page))
    assert full.status.item() == 0
    _close(out, ref, dtype, 3.0)
    # what the cache holds: the normed keys and the values, biases included, zeros beyond their sizes
    k = full.read(0, full.k_pool, n).float().cpu()
    v = full.read(0, full.v_pool, n).float().cpu()
    _close(k[..., :dim], plain.rms((_cpu(x).double() @ w["k"].double().T).float().add(w["k.b"]).view(n, kv, dim), 1e-5) * w["k.norm"], dtype, 2.0)
    _close(v[..., :vdim], ((_cpu(x).double() @ w["v"].double().T).float() + w["v.b"]).view(n, kv, vdim), dtype, 2.0)
    assert (k[..., dim:] == 0).all() and (v[..., vdim:] == 0).all()
    full, _ = _ctx([(0, n)], page, kv, att.cache_dim, dtype, seed=2)
    _close(_kv_portions(att, x, (page + 3, 2, 13, 2) + (1,) * n, page, dtype, full), ref, dtype, 3.0)
    # two unequal requests in one step (the second decodes a token behind what an earlier step left)
    both_pb, _ = _ctx([(0, 30), (0, n)], page, kv, att.cache_dim, dtype, seed=7)
    view = KVEntryView(0, both_pb.k_pool, both_pb.v_pool, page)
    _, warm = _ctx([(0, 1), (0, n - 1)], page, kv, att.cache_dim, dtype, share=both_pb)
    att.forward(torch.cat((x[:1], x[:n - 1])).contiguous(), warm, view)
    _, ctx = _ctx([(0, 30), (n - 1, 1)], page, kv, att.cache_dim, dtype, share=both_pb)
    both = att.forward(torch.cat((x[:30], x[n - 1:])).contiguous(), ctx, view)
    _close(both[:30], ref[:30], dtype, 3.0)
    _close(both[30:], ref[n - 1:], dtype, 3.0)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n, dim, heads, kv", [(700, 32, 4, 2), (1900, 128, 4, 2), (1300, 96, 8, 1)])
def test_attention_finds_a_far_key_among_hundreds(dtype, n, dim, heads, kv):
    """The last query and one earlier token are made so that this pair scores far above everything else (the query matrix is
    the key matrix, so a token scores itself as high; the two split the weight): the earlier token's value must show wherever it
    lies: the first token, the last and the first of a page, the middle."""
    att, m = _attention(dtype, heads, kv, dim, 32, scale=24.0 / dim, coef=0.3, every=64)

    def needle(t):
        t["q"].copy_(t["k"].view(kv, 1, dim, HIDDEN).expand(kv, heads // kv, dim, HIDDEN).reshape(heads * dim, HIDDEN))
        t["q.b"].zero_()
        t["k.b"].zero_()
        t["k.norm"].fill_(1.0)
        t["q.norm"].fill_(1.0)

    w = _bind(att, dtype, change=needle)
    last = n - 1
    direction = _x(1, dtype, 3.0)[0]
    base = _x(n, dtype, 1.0)
    for at in (0, 15, 16, n // 2):
        x = base.clone()
        x[last] = direction
        x[at] = direction + _x(1, dtype, 0.3)[0]
        ref = _attention_ref(x, w, m)
        blank = x.clone()
        blank[at] = base[at]
        assert (ref[last] - _attention_ref(blank, w, m)[last]).abs().max() > 0.02, "the test's needle does not show"
        full, _ = _ctx([(0, n)], 16, kv, att.cache_dim, dtype, seed=3)
        view = KVEntryView(0, full.k_pool, full.v_pool, 16)
        _, ctx = _ctx([(0, n)], 16, kv, att.cache_dim, dtype, share=full)
        _close(att.forward(x, ctx, view), ref, dtype, 3.0)  # in a prompt
        _, ctx = _ctx([(last, 1)], 16, kv, att.cache_dim, dtype, share=full)
        _close(att.forward(x[last:].contiguous(), ctx, view), ref[last:], dtype, 3.0)  # decoded alone over the same pages
        _, ctx = _ctx([(n - 3, 3)], 16, kv, att.cache_dim, dtype, share=full)
        _close(att.forward(x[n - 3:].contiguous(), ctx, view), ref[n - 3:], dtype, 3.0)  # a short portion


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dim", [16, 128])
def test_sink_empties_a_head_whose_scores_are_low(dtype, dim):
    """Keys that all score far below the sink's zero leave an output of nearly nothing; without the sink the weights would sum to
    one. The first token of a sequence has one key and the sink."""
    att, m = _attention(dtype, 2, 1, dim, 16, scale=1.0 / dim, coef=0.0, every=8)

    def low(t):
        t["k.b"].fill_(1.0)
        t["k"].mul_(0.05)
        t["q"].mul_(0.05)
        t["q.b"][:dim], t["q.b"][dim:] = -1.0, 1.0  # head 0 scores about -9, head 1 about +9
        t["q.norm"].fill_(3.0)
        t["k.norm"].fill_(3.0)
        t["o"].copy_(torch.eye(HIDDEN, 32))

    w = _bind(att, dtype, change=low)
    n = 20
    x = _x(n, dtype)
    ref = _attention_ref(x, w, m)
    full, ctx = _ctx([(0, n)], 8, 1, att.cache_dim, dtype)
    view = KVEntryView(0, full.k_pool, full.v_pool, 8)
    out = att.forward(x, ctx, view)
    _close(out, ref, dtype, 3.0)
    assert out[:, :16].abs().max() < 0.05 * out[:, 16:32].abs().max()
    _, ctx = _ctx([(n - 1, 1)], 8, 1, att.cache_dim, dtype, share=full)
    _close(att.forward(x[n - 1:].contiguous(), ctx, view), ref[n - 1:], dtype, 3.0)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("every, coef", [(1, 0.5), (8, 2.0), (100, -0.3), (2.5, 0.7)])
def test_query_temperature_by_position(dtype, every, coef):
    """A large scale makes the temperature decide between two keys that nearly tie: the outputs follow the oracle's on both
    sides of every multiple, in a prompt and decoded, and differ from those without a temperature."""
    att, m = _attention(dtype, 2, 1, 16, 16, scale=0.5, coef=coef, every=every)
    w = _bind(att, dtype, change=lambda t: t["q.norm"].mul_(1.5))
    n = 230
    x = _x(n, dtype)
    ref = _attention_ref(x, w, m)
    without = {k: v for k, v in m.items() if k != "q_temp"}
    assert (plain.attention(_cpu(x), w, "", without, 1e-5, torch.float32) - ref)[every > 99 and 101 or 9:].abs().max() > 0.02
    full, ctx = _ctx([(0, n)], 16, 1, att.cache_dim, dtype)
    view = KVEntryView(0, full.k_pool, full.v_pool, 16)
    _close(att.forward(x, ctx, view), ref, dtype, 3.0)
    for at in (0, 6, 7, 8, 15, 16, 98, 99, 100, 199, n - 1):
        _, ctx = _ctx([(at, 1)], 16, 1, att.cache_dim, dtype, share=full)
        _close(att.forward(x[at:at + 1].contiguous(), ctx, view), ref[at:at + 1], dtype, 3.0)


# --------------------------------------------------------------------------- matrix memory
def _memory(dtype, heads, dim, vdim, cap):
    from miniserve_b200.models.vumedra import _mlstm as spec_of

    m = vx.memory_layer(heads, dim, vdim, cap)["mixer"]
    return build_part("mixer", spec_of(HIDDEN, 1e-5, m), BuildEnv(dtype, DEV)), m


def _memory_weights(t):
    h = t["f.b"].numel()
    t["f.b"].copy_(torch.linspace(-1.0, 5.0, h) if h > 1 else torch.tensor([3.0]))
    t["i"].mul_(2.0)
    t["f"].mul_(2.0)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, dim, vdim, cap", [(3, 16, 24, 12.0), (5, 12, 20, 7.5), (1, 24, 16, 3.0), (4, 64, 96, 20.0), (2, 128, 40, 15.0), (1, 8, 8, 1.0),
                                                   (2, 36, 260, 10.0), (2, 128, 256, 15.0), (1, 256, 136, 8.0), (3, 40, 200, 9.0)])
def test_matrix_memory_whole_in_portions_and_decoded(dtype, heads, dim, vdim, cap):
    part, m = _memory(dtype, heads, dim, vdim, cap)
    w = _bind(part, dtype, change=_memory_weights)
    n = 70
    x = _x(n, dtype)
    ref = plain.mlstm(_cpu(x), w, "", m, 1e-5, torch.float32)
    noise = None
    if dtype == torch.bfloat16:
        noise = (plain.mlstm(_cpu(x), w, "", m, 1e-5, dtype) - ref).abs().amax(dim=1)
    views = _state_views(part)
    _close(_state_portions(part, views, x, (n,), 1, dtype), ref, dtype, 3.0, noise)
    # the same slot again; single tokens from the very first one, then portions down to two tokens, then token by token
    _close(_state_portions(part, views, x, (1, 1, 2, 1, 3, 2, 17, 2, 9) + (1,) * n, 1, dtype), ref, dtype, 3.0, noise)
    _, ctx = _ctx([(0, 21), (0, n - 9)], dtype=dtype, slots=[4, 0])
    both = part.forward(torch.cat((x[:21], x[:n - 9])), ctx, views)
    _close(both, torch.cat((ref[:21], ref[:n - 9])), dtype, 3.0, None if noise is None else torch.cat((noise[:21], noise[:n - 9])))
    _, ctx = _ctx([(n - 9, 1), (21, 30)], dtype=dtype, slots=[0, 4])
    both = part.forward(torch.cat((x[n - 9:n - 8], x[21:51])), ctx, views)
    _close(both, torch.cat((ref[n - 9:n - 8], ref[21:51])), dtype, 3.0, None if noise is None else torch.cat((noise[n - 9:n - 8], noise[21:51])))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, dim, vdim", [(2, 16, 24), (4, 64, 64), (1, 400, 16), (2, 128, 256)])
def test_matrix_memory_over_a_long_portion_and_long_decoding(dtype, heads, dim, vdim):
    """Portions of hundreds of tokens (the walk may be cut into segments), behind an earlier portion, beside a short row, and
    hundreds of tokens decoded one by one from the state they left."""
    part, m = _memory(dtype, heads, dim, vdim, 12.0)
    w = _bind(part, dtype, change=_memory_weights)
    n = 1000
    x = _x(n, dtype)
    run = torch.float32 if dtype == torch.float32 else dtype
    ref = plain.mlstm(_cpu(x), w, "", m, 1e-5, torch.float32, acc=torch.float64)
    noise = (plain.mlstm(_cpu(x), w, "", m, 1e-5, run) - ref).abs().amax(dim=1)
    views = _state_views(part)
    _close(_state_portions(part, views, x[:700], (700,), 1, dtype), ref[:700], dtype, 3.0, noise[:700])
    _close(_state_portions(part, views, x, (37, 663) + (1,) * n, 2, dtype), ref, dtype, 3.0, noise)
    _, ctx = _ctx([(0, 5), (0, 690)], dtype=dtype, slots=[4, 0])
    both = part.forward(torch.cat((x[:5], x[:690])), ctx, views)
    _close(both, torch.cat((ref[:5], ref[:690])), dtype, 3.0, torch.cat((noise[:5], noise[:690])))


@pytest.mark.parametrize("dtype", DTYPES)
def test_matrix_memory_when_the_running_maximum_jumps(dtype):
    """Input gates at both caps in turn and forget gates that shut: the maximum jumps up by twice the cap and decays back to below
    zero, so the state is rescaled by both exponentials and the denominator's floor exp(-m) takes over and gives way again."""
    part, m = _memory(dtype, 2, 16, 16, 14.0)

    def jumps(t):
        t["i"].zero_()
        t["f"].zero_()
        t["i"][:, 0], t["f"][:, 1] = 100.0, 100.0  # input channel 0 drives the input gate, channel 1 the forget gate
        t["i.b"].zero_()
        t["f.b"].zero_()
        t["q"][:, :2], t["k"][:, :2], t["v"][:, :2] = 0.0, 0.0, 0.0

    w = _bind(part, dtype, change=jumps)
    n = 90
    x = _x(n, dtype)
    i = torch.zeros(n)
    f = torch.zeros(n)
    for t in range(n):
        i[t] = (1.0, -1.0, -1.0, 0.0, 0.02, -0.5)[(t // 5) % 6]
        f[t] = (0.05, 1.0, -0.02, 0.3)[(t // 7) % 4]
    x[:, 0], x[:, 1] = i.to(DEV).to(dtype), f.to(DEV).to(dtype)
    ref = plain.mlstm(_cpu(x), w, "", m, 1e-5, torch.float32, acc=torch.float64)
    noise = (plain.mlstm(_cpu(x), w, "", m, 1e-5, dtype) - ref).abs().amax(dim=1)
    views = _state_views(part)
    _close(_state_portions(part, views, x, (n,), 0, dtype), ref, dtype, 3.0, noise)
    _close(_state_portions(part, views, x, (2, 31, 2) + (1,) * n, 3, dtype), ref, dtype, 3.0, noise)


@pytest.mark.parametrize("dtype", DTYPES)
def test_matrix_memory_keeps_an_early_token_through_an_open_forget_gate(dtype):
    """Head 0 hardly forgets and head 1 forgets within a few tokens: a change of the first token's input must show in the last
    token's output through head 0's channels, and not through head 1's."""
    part, m = _memory(dtype, 2, 16, 16, 10.0)

    def gates(t):
        t["f"].zero_()
        t["f.b"].copy_(torch.tensor([9.0, -3.0]))
        t["i"].zero_()

    w = _bind(part, dtype, change=gates)
    n = 90
    x = _x(n, dtype)
    other = x.clone()
    other[0] = _x(1, dtype, 4.0)[0]
    views = _state_views(part)
    feats = []
    for inp in (x, other):
        _, ctx = _ctx([(0, n - 1)], dtype=dtype, slots=[3])
        part.forward(inp[:n - 1].contiguous(), ctx, views)
        _, ctx = _ctx([(n - 1, 1)], dtype=dtype, slots=[3])
        f = torch.zeros(1, part.feature_width, device=DEV, dtype=dtype)
        part.features(inp[n - 1:].contiguous(), ctx, views, f)
        feats.append(f.float().cpu()[0])
    diff = (feats[0] - feats[1]).abs()
    assert diff[:16].max() > 2e-2 and diff[16:].max() < 1e-3
    _, ctx = _ctx([(0, n)], dtype=dtype, slots=[0])
    ref = plain.mlstm(_cpu(other), w, "", m, 1e-5, torch.float32)
    noise = (plain.mlstm(_cpu(other), w, "", m, 1e-5, dtype) - ref).abs().amax(dim=1)
    _close(part.forward(other, ctx, views), ref, dtype, 3.0, noise)


@pytest.mark.parametrize("heads, groups, dk, dv, ones", [(2, 2, 128, 256, True), (4, 2, 64, 96, False), (3, 3, 8, 8, True), (2, 1, 256, 136, True), (1, 1, 40, 200, False)])
def test_decay_rule_over_chunks_on_the_tensor_cores(heads, groups, dk, dv, ones):
    """Rows from one token to several chunks, some behind an earlier state, decays from one to zero, against the recurrence in
    64-bit: the tensor cores see what is not exact in bfloat16 as two numbers, so the error stays far below bfloat16's."""
    from miniserve_b200 import ops

    rows = [(0, 1), (5, 64), (0, 65), (300, 200), (0, 7), (9, 1), (0, 129)]
    _, ctx = _ctx(rows, dtype=torch.bfloat16, slots=[6, 0, 3, 1, 4, 5, 2])
    t = sum(n for _, n in rows)
    q, k = (torch.randn(t, groups * dk, device=DEV).bfloat16() for _ in range(2))
    v = torch.randn(t, heads * dv, device=DEV).bfloat16()
    decay = torch.rand(t, heads, device=DEV) ** 0.05
    decay[::17] = 0.0
    decay[5::29] = 1.0
    decay[70:100] = 1e-20
    write = torch.rand(t, heads, device=DEV) * 3
    extra = int(ones)
    state = torch.randn(7, heads, dv + extra, dk, device=DEV)
    held = state.clone()
    o = torch.full((t, heads, dv + 4), float("nan"), device=DEV)
    assert ops.chunk_scan_ok(q, k, v, dk, dv, ctx)
    ops.chunk_scan(o, state, q, k, v, decay, write, ctx, heads, dk, dv, 0.25, ones)
    qd, kd, vd, ad, wd = (x.double().cpu() for x in (q, k, v, decay, write))
    vd = vd.view(t, heads, dv)
    if ones:
        vd = torch.cat((vd, torch.ones(t, heads, 1, dtype=torch.float64)), -1)
    head_group = [h // (heads // groups) for h in range(heads)]
    qh, kh = qd.view(t, groups, dk)[:, head_group], kd.view(t, groups, dk)[:, head_group]
    at = 0
    for (start, n), slot in zip(rows, ctx.state_slot.tolist()):
        s = held[slot].double().cpu() if start else torch.zeros(heads, dv + extra, dk, dtype=torch.float64)
        for i in range(at, at + n):
            s = ad[i][:, None, None] * s + wd[i][:, None, None] * vd[i][:, :, None] * kh[i][:, None, :]
            want = (s * qh[i][:, None, :]).sum(-1) * 0.25
            size = (s.abs() * qh[i].abs()[:, None, :]).sum(-1) * 0.25 + 1e-3
            assert ((o[i, :, :dv + extra].double().cpu() - want).abs() / size).max() < 6e-5, (slot, i - at)
        assert (state[slot].double().cpu() - s).abs().max() < 3e-5 * max(1.0, s.abs().max().item())
        at += n


# --------------------------------------------------------------------------- gated linear recurrence
def _recurrent(dtype, width, blocks, conv):
    from miniserve_b200.models.vumedra import _rglru as spec_of

    m = vx.recurrent_layer(width, blocks, conv)["mixer"]
    return build_part("mixer", spec_of(HIDDEN, 1e-5, m), BuildEnv(dtype, DEV)), m


def _recurrent_weights(t):
    t["lam"].copy_(torch.linspace(-7.0, 1.0, t["lam"].numel()))  # from hundreds of tokens to one
    t["conv"].mul_(2.0)


RECURRENT_CASES = [(48, 3, 4), (28, 4, 2), (36, 1, 1), (80, 5, 3), (256, 2, 4), (7, 7, 5), (40, 8, 9), (160, 2, 4)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width, blocks, conv", RECURRENT_CASES)
def test_gated_recurrence_whole_in_portions_and_decoded(dtype, width, blocks, conv):
    part, m = _recurrent(dtype, width, blocks, conv)
    w = _bind(part, dtype, change=_recurrent_weights)
    n = 70
    x = _x(n, dtype)
    ref = plain.rglru(_cpu(x), w, "", m, 1e-5, torch.float32)
    views = _state_views(part)
    _close(_state_portions(part, views, x, (n,), 1, dtype), ref, dtype, 3.0)
    # the same slot again; portions shorter than the convolution's history, single tokens from the very first one
    _close(_state_portions(part, views, x, (1, 1, 2, 1, 3, 2, 17, 2, 9) + (1,) * n, 1, dtype), ref, dtype, 3.0)
    _close(_state_portions(part, views, x, (2,) * n, 2, dtype), ref, dtype, 3.0)
    _, ctx = _ctx([(0, 21), (0, n - 9)], dtype=dtype, slots=[4, 0])
    both = part.forward(torch.cat((x[:21], x[:n - 9])), ctx, views)
    _close(both, torch.cat((ref[:21], ref[:n - 9])), dtype, 3.0)
    _, ctx = _ctx([(n - 9, 1), (21, 30)], dtype=dtype, slots=[0, 4])
    both = part.forward(torch.cat((x[n - 9:n - 8], x[21:51])), ctx, views)
    _close(both, torch.cat((ref[n - 9:n - 8], ref[21:51])), dtype, 3.0)
    # two decoding rows in one step
    _, ctx = _ctx([(n - 8, 1), (51, 1)], dtype=dtype, slots=[0, 4])
    both = part.forward(torch.cat((x[n - 8:n - 7], x[51:52])), ctx, views)
    _close(both, torch.cat((ref[n - 8:n - 7], ref[51:52])), dtype, 3.0)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width, blocks", [(48, 3), (256, 2)])
def test_gated_recurrence_over_long_portions_and_long_decoding(dtype, width, blocks):
    """Portions of every form that the walk has: one CTA, two and eight per row, several passes (1,300 tokens), behind an
    earlier portion, beside a row of five tokens and one decoding row, then hundreds of tokens one by one."""
    part, m = _recurrent(dtype, width, blocks, 4)
    w = _bind(part, dtype, change=_recurrent_weights)
    n = 1500
    x = _x(n, dtype)
    ref = plain.rglru(_cpu(x), w, "", m, 1e-5, torch.float32)
    views = _state_views(part)
    _close(_state_portions(part, views, x[:1300], (1300,), 1, dtype), ref[:1300], dtype, 3.0)
    _close(_state_portions(part, views, x, (37, 130, 63, 64, 65, 600, 2, 239) + (1,) * n, 2, dtype), ref, dtype, 3.0)
    _, ctx = _ctx([(1300, 1), (0, 5), (0, 690)], dtype=dtype, slots=[1, 4, 0])
    out = part.forward(torch.cat((x[1300:1301], x[:5], x[:690])), ctx, views)
    _close(out, torch.cat((ref[1300:1301], ref[:5], ref[:690])), dtype, 3.0)


@pytest.mark.parametrize("dtype", DTYPES)
def test_gated_recurrence_remembers_through_a_slow_channel(dtype):
    part, m = _recurrent(dtype, 32, 2, 2)

    def decays(t):
        t["lam"].copy_(torch.cat((torch.full((16,), -9.0), torch.full((16,), 1.0))))
        t["y"].zero_()
        t["y.b"].fill_(2.0)

    w = _bind(part, dtype, change=decays)
    n = 90
    x = _x(n, dtype)
    other = x.clone()
    other[0] = _x(1, dtype, 4.0)[0]
    views = _state_views(part)
    feats = []
    for inp in (x, other):
        _, ctx = _ctx([(0, n - 1)], dtype=dtype, slots=[3])
        part.forward(inp[:n - 1].contiguous(), ctx, views)
        _, ctx = _ctx([(n - 1, 1)], dtype=dtype, slots=[3])
        f = torch.zeros(1, part.width, device=DEV, dtype=dtype)
        part.features(inp[n - 1:].contiguous(), ctx, views, f)
        feats.append(f.float().cpu()[0])
    diff = (feats[0] - feats[1]).abs()
    assert diff[:16].max() > 1e-2 and diff[16:].max() < 1e-3
    _, ctx = _ctx([(0, n)], dtype=dtype, slots=[0])
    _close(part.forward(other, ctx, views), plain.rglru(_cpu(other), w, "", m, 1e-5, torch.float32), dtype, 3.0)


# --------------------------------------------------------------------------- feed-forward
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("hidden, ff, experts, top, shared", [
    (48, 24, 6, 2, 40), (36, 20, 5, 1, 28), (40, 12, 1, 1, 0), (64, 64, 8, 4, 96), (56, 24, 3, 3, 0), (128, 136, 30, 8, 72), (48, 20, 12, 6, 44)])
def test_router_and_experts(dtype, hidden, ff, experts, top, shared):
    from miniserve_b200.models.vumedra import _feed_forward as spec_of

    mlp = vx.moe(ff, experts, top, shared)
    ffn = build_part("feed_forward", spec_of(hidden, mlp), BuildEnv(dtype, DEV))
    w = _bind(ffn, dtype, change=lambda t: t["router"].mul_(1.5))
    for n in (1, 2, 77, 300):
        x = torch.randn(n, hidden, device=DEV).to(dtype)
        _, ctx = _ctx([(0, n)], dtype=dtype)
        idx, wgt = ffn.route(x, ctx)
        chosen, weights = plain.route(_cpu(x), w, "", top, torch.float32)
        order_g, order_w = idx.long().cpu().sort(-1), chosen.sort(-1)
        assert (order_g.values == order_w.values).all()
        # the expert is of degree two in its input: the part hands on the square of the weight that multiplies the input
        assert torch.allclose(wgt.cpu().gather(1, order_g.indices), weights.gather(1, order_w.indices) ** 2, rtol=1e-4, atol=1e-6)
        want = plain.moe_ff(_cpu(x), w, "", mlp, torch.float32)
        _close(ffn.forward(x, ctx), want, dtype, 3.0)
        if dtype == torch.bfloat16:  # the products on the older tensor-core path too (what shapes off the tcgen05 kernel's take)
            from miniserve_b200.ops import experts as xo

            held, xo.TC_EXPERTS = xo.TC_EXPERTS, False
            try:
                _close(ffn.forward(x, ctx), want, dtype, 3.0)
            finally:
                xo.TC_EXPERTS = held


def test_scores_are_sigmoids_and_are_not_renormalised():
    """Router rows of zero but for the biggest input: scores 1/2 everywhere but for two; the weights' squares come back."""
    from miniserve_b200.models.vumedra import _feed_forward as spec_of

    ffn = build_part("feed_forward", spec_of(HIDDEN, vx.moe(24, 4, 2, 0)), BuildEnv(torch.float32, DEV))

    def rows(t):
        t["router"].zero_()
        t["router"][1, 0], t["router"][3, 0] = 1.0, 2.0

    _bind(ffn, torch.float32, change=rows)
    x = torch.zeros(1, HIDDEN, device=DEV)
    x[0, 0] = 1.0
    _, ctx = _ctx([(0, 1)])
    idx, wgt = ffn.route(x, ctx)
    assert idx.tolist() == [[3, 1]]
    want = torch.tensor([[1 / (1 + math.exp(-2)), 1 / (1 + math.exp(-1))]]) ** 2
    assert torch.allclose(wgt.cpu(), want, rtol=1e-6)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("hidden, inter", [(40, 72), (36, 52)])
def test_dense_feed_forward(dtype, hidden, inter):
    from miniserve_b200.models.vumedra import _feed_forward as spec_of

    ffn = build_part("feed_forward", spec_of(hidden, vx.dense(inter)), BuildEnv(dtype, DEV))
    w = _bind(ffn, dtype)
    for n in (9, 40):
        x = (torch.randn(n, hidden, device=DEV) * 2).to(dtype)
        _, ctx = _ctx([(0, n)], dtype=dtype)
        _close(ffn.forward(x, ctx), plain.dense_ff(_cpu(x), w, "", torch.float32), dtype, 3.0)


# --------------------------------------------------------------------------- whole models
@pytest.fixture(scope="module", params=["a", "b", "c", "d"])
def model(request, tmp_path_factory):
    raw = getattr(vx, "config_" + request.param)()
    folder = vx.write_model(tmp_path_factory.mktemp("vumedra_" + request.param), raw, seed=ord(request.param))
    return dict(folder=folder, raw=raw, oracle=vx.oracle(folder), rounded=vx.oracle(folder, torch.bfloat16),
                page=dict(a=16, b=8, c=32, d=16)[request.param])


def _logits_close(model, dtype, got, ids, what=""):
    """32-bit: within F32 of the oracle. bfloat16: as near as rounding allows, position by position (``vx.rounded_ok``)."""
    want = model["oracle"](ids)
    if dtype == "float32":
        ok, report = vx.float32_ok(model["folder"], got, want, ids, F32)
        assert ok, f"{what}: {report}"
    else:
        ok, report = vx.rounded_ok(got, want, model["rounded"](ids))
        assert ok, f"{what}: {report}"


def test_layer_streams_in_float32(model):
    """The residual stream after every layer, against the oracle's."""
    from miniserve_b200.cache import CacheManager
    from miniserve_b200.engine.loader import load_model
    from miniserve_b200.engine.step import StepFunction, StepRow

    ids = _ids(29, model["raw"]["vocab"], 8)
    want = vx.layer_streams(model["folder"], ids)
    _, _, net = load_model(model["folder"], "float32", "cuda:0")
    cache = CacheManager(net.entry_caches, 8, 16, 2, dtype=net.dtype, device=net.device)
    ctx = StepFunction(net, cache).prepare([StepRow(cache.new_request(), ids, [0])])
    stream = ResidualStream(net.embed(ctx, cache.entry_views))
    for i, e in enumerate(net.spec.run_order):
        stream = net.layers[e.layer].forward(stream, ctx, cache.entry_views[i])
        norm = stream.pending_norm
        x = stream.total.double().cpu() + plain.rms(_cpu(stream.pending), norm.eps).double() * norm.float_weight.item()
        assert (x - want[i].double()).abs().max() < 1e-4 * max(1.0, want[i].abs().max().item()), f"after layer {i}"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_whole_decoded_and_in_portions(model, dtype):
    vocab = model["raw"]["vocab"]
    run = vx.Runner(model["folder"], dtype, max_tokens=256, page_size=model["page"])
    for n, seed in ((1, 1), (2, 2), (37, 3), (150, 4)):
        ids = _ids(n, vocab, seed)
        _logits_close(model, dtype, run.feed("w", ids, [n]), ids, f"{n} whole")
        if n > 2:
            _logits_close(model, dtype, run.feed("d", ids, [n - min(n - 1, 110), 1]), ids, f"{n} decoded")
            _logits_close(model, dtype, run.feed("c", ids, [7, 2, 24, 3, model["page"], 2, 5, 31, 2, 1, 1, 2, 9]), ids, f"{n} in portions")
        assert run.cache.is_idle()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_mixed_batches_reuse_pages_and_slots(model, dtype):
    """Up to four live requests, portions of some beside single tokens of others, a pool that holds only what is live and
    four state slots: every page and slot is used by several requests in turn (pages are filled with NaN when given back)."""
    vocab = model["raw"]["vocab"]
    seqs = {f"r{i}": _ids(n, vocab, 20 + i) for i, n in enumerate([90, 5, 64, 33, 1, 120, 17, 48, 2, 75])}
    run = vx.Runner(model["folder"], dtype, max_tokens=4 * 128, page_size=model["page"], max_requests=4)
    rng = random.Random(5)
    waiting, live, at, got = list(seqs), [], {}, {k: [] for k in seqs}
    while waiting or live:
        while waiting and len(live) < 4:
            live.append(waiting.pop(0))
            at[live[-1]] = 0
        entries, ended = [], []
        order = sorted(live, key=lambda r: at[r] == 0 or len(seqs[r]) - at[r] > 40)  # decoding rows first
        for rid in order:
            left = len(seqs[rid]) - at[rid]
            n = 1 if left <= 40 and at[rid] > 0 else min(left, rng.choice([2, 3, 16, 29, 50]))
            if rng.random() < 0.15 and len(order) > 1:
                continue  # left out of this step
            entries.append((rid, seqs[rid][at[rid]:at[rid] + n], "all"))
            at[rid] += n
            if at[rid] == len(seqs[rid]):
                ended.append(rid)
        if not entries:
            continue
        logits = run.step(entries, end=ended)
        i = 0
        for rid, toks, _ in entries:
            got[rid].append(logits[i:i + len(toks)])
            i += len(toks)
        live = [r for r in live if r not in ended]
    for rid in seqs:
        _logits_close(model, dtype, torch.cat(got[rid]), seqs[rid], rid)
    assert run.cache.is_idle()


def test_long_decoding_in_float32(model):
    ids = _ids(400, model["raw"]["vocab"], 9)
    run = vx.Runner(model["folder"], "float32", max_tokens=448, page_size=model["page"])
    _logits_close(model, "float32", run.feed("long", ids, [3, 1]), ids)


def test_a_long_prompt_whole_and_in_two_portions(model):
    ids = _ids(1200, model["raw"]["vocab"], 10)
    run = vx.Runner(model["folder"], "float32", max_tokens=1216, page_size=model["page"])
    _logits_close(model, "float32", run.feed("w", ids, [1200]), ids, "whole")
    _logits_close(model, "float32", run.feed("c", ids, [513, 2, 685]), ids, "in portions")


def test_trace_runner_replays_a_schedule(model, tmp_path):
    from tests.trace_util import Trace, run_trace

    vocab = model["raw"]["vocab"]
    a, b = _ids(50, vocab, 31), _ids(21, vocab, 32)
    tr = Trace()
    tr.step([("a", a[:30], [0, 29])])
    tr.step([("a", a[30:31], [0]), ("b", b[:19], "last")])
    tr.step([("b", b[19:20], [0]), ("a", a[31:], "all")], end=["a"])
    tr.step([("b", b[20:], [0])], end=["b"])
    tr.step([("c", b, "last")], end=["c"])  # in the pages and the slot that were given back
    out = run_trace(model["folder"], "float32", tr, tmp_path / "out", page_size=model["page"], vocab=vocab)
    want = {"a": model["oracle"](a), "b": model["oracle"](b), "c": model["oracle"](b)}
    assert len(out) == 2 + 2 + 1 + 19 + 1 + 1
    ids = {"a": a, "b": b, "c": b}
    for rid in want:
        rows = sorted((pos, logits) for (r, pos, _), logits in out.items() if r == rid)
        got = want[rid].clone()
        for pos, logits in rows:
            got[pos] = logits
        _logits_close(model, "float32", got, ids[rid], rid)


@pytest.mark.parametrize("dtype, cuda_graph", [("float32", False), ("float32", True), ("bfloat16", True)])
def test_greedy_generation_through_the_entry_point(model, dtype, cuda_graph):
    from miniserve_b200.engine import LLM, SamplingParams

    vocab = model["raw"]["vocab"]
    prompts = [_ids(n, vocab, 40 + n) for n in (5, 17, 33, 1, 9, 70)]
    llm = LLM(model["folder"], dtype=dtype, kv_pool_tokens=1024, page_size=model["page"], max_running=4,
              chunked_prefill_size=24, cuda_graph=cuda_graph)
    outs = llm.generate(prompts, SamplingParams(max_new_tokens=10))
    assert llm.engine.cache.is_idle()
    for p, o in zip(prompts, outs):
        assert len(o) == 10
        every = model["oracle"](list(p) + list(o))  # causal: row i is what the oracle says after tokens 0..i
        # bfloat16: how far rounding alone moves the oracle's own logits at each position
        moved = (model["rounded"](list(p) + list(o)) - every).abs().amax(dim=1) if dtype == "bfloat16" else None
        for i, t in enumerate(o):  # teacher-forced: each chosen token is the oracle's best, or within rounding of it
            at = len(p) + i - 1
            logits = every[at]
            slack = 1e-4 if dtype == "float32" else max(0.15, 3.0 * moved[at].item())
            assert (logits.max() - logits[t]).item() <= slack, (at + 1, t)


def test_generation_survives_preemption(model):
    """A pool too small for what is admitted: requests are sent back and start over, their state with them."""
    from miniserve_b200.engine import LLM, SamplingParams

    if not any(layer["type"] == "attention" for layer in model["raw"]["layers"]):
        pytest.skip("no pages: nothing runs out")
    vocab = model["raw"]["vocab"]
    prompts = [_ids(n, vocab, 60 + n) for n in (30, 41, 28)]
    llm = LLM(model["folder"], dtype="float32", kv_pool_tokens=160, page_size=model["page"], max_running=4, chunked_prefill_size=64)
    outs = llm.generate(prompts, SamplingParams(max_new_tokens=30))
    assert llm.engine.scheduler.num_preemptions > 0 and llm.engine.cache.is_idle()
    for p, o in zip(prompts, outs):
        every = model["oracle"](list(p) + list(o))
        for i, t in enumerate(o):
            logits = every[len(p) + i - 1]
            assert (logits.max() - logits[t]).item() <= 1e-4
