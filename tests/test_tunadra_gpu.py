"""Tunadra on the GPU against the plain implementation: each mechanism alone, whole prompts against
token-by-token decoding and portions down to two tokens, unequal requests in one batch against each
alone, pages and state slots that are given back and used again, keys far away and at page borders (in
prompts and in decoding), the first tokens of a sequence, long decoding, sizes that are no round numbers,
the trace runner and greedy generation through the entry point."""

import math
import random

import pytest
import torch

from miniserve_b200 import ops
from miniserve_b200.cache.manager import KVEntryView, StateEntryView
from miniserve_b200.config import PartSpec
from miniserve_b200.ops import experts as xo
from miniserve_b200.ops import native
from miniserve_b200.parts import BuildEnv, ResidualStream, build_part
from miniserve_b200.parts.block import StreamLinks
from tests import tunadra_util as tx
from tests.kernel_util import PagedBatch, make_context
from tests.plain import tunadra_plain as plain

pytestmark = pytest.mark.gpu
DEV = torch.device("cuda")
F32 = 1e-4  # logits in 32-bit: distance over their spread (rel_err); the oracle sums its products in 64-bit, the engine in 32-bit
DTYPES = [torch.float32, torch.bfloat16]
HIDDEN = 48


def _ids(n, vocab, seed):
    rng = random.Random(seed)
    return [rng.randrange(vocab) for _ in range(n)]


def _close(got, want, dtype, scale=1.0, noise=None):
    """``noise`` [T]: what rounding alone costs the plain form at each token; a token may be four times that far on top of the tolerance."""
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
    torch.manual_seed(8642)
    torch.cuda.manual_seed(8642)


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


# --------------------------------------------------------------------------- embedding, head
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width, scale", [(64, 3.5), (45, 0.25), (36, 1.0), (1024, 12.5)])
def test_scaled_embedding_with_a_sinusoid(dtype, width, scale):
    emb = build_part("embedding", PartSpec("summed_embedding", dict(vocab=61, hidden=width, name="embed", sinusoid=10000.0, scale=scale)), BuildEnv(dtype, DEV))
    w = _bind(emb, dtype, std=1.0)
    assert emb.cache_need() is None
    raw = tx.config([], width=width, vocab=61, scale=scale)
    ids = _ids(70, 61, 1)
    want = plain.embed(raw, w, ids)
    _, ctx = _ctx([(0, 70)], ids=ids)
    _close(emb.forward(ctx), want, torch.float32)
    _, ctx = _ctx([(33, 1), (0, 5)], ids=[ids[33]] + ids[:5])  # a decoded token beside a prompt: the position decides, not the place
    _close(emb.forward(ctx), torch.cat((want[33:34], want[:5])), torch.float32)


@pytest.mark.parametrize("cap", [0.5, 30.0])
@pytest.mark.parametrize("vocab", [96, 97])
def test_capped_logits(cap, vocab):
    head = build_part("head", PartSpec("linear_head", dict(vocab=vocab, hidden=HIDDEN, name="head", softcap=cap)), BuildEnv(torch.float32, DEV))
    w = _bind(head, torch.float32, std=3.0)
    x = _x(5, torch.float32, 2.0)
    _, ctx = _ctx([(0, 5)])
    want = plain.softcap(_cpu(x) @ w["head"].T, cap)
    assert want.abs().max() > 0.9 * cap
    _close(head.forward(x, ctx), want, torch.float32)


# --------------------------------------------------------------------------- several streams
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [36, 45, 64, 1024, 2056, 4104, 9001])
@pytest.mark.parametrize("count", [1, 2, 3, 4, 7])
def test_streams_norm_and_update(dtype, width, count):
    env = BuildEnv(dtype, DEV)
    norm = build_part("norm", PartSpec("rmsnorm", dict(size=width, eps=1e-5, name="g")), env)
    wn = _bind(norm, dtype)["g"]
    a, b = StreamLinks(PartSpec("stream_links", dict(streams=count)), env), StreamLinks(PartSpec("stream_links", dict(streams=count)), env)
    wa, wb = _bind(a, dtype, seed=3, std=0.6), _bind(b, dtype, seed=4, std=0.6)
    n = 6
    x0 = torch.randn(n, width, device=DEV) * 2
    y1, y2 = ((torch.randn(n, width, device=DEV) * s).to(dtype) for s in (1.0, 0.3))
    streams = _cpu(x0)[:, None, :].repeat(1, count, 1)
    h = lambda u: plain.rms(u, 1e-5) * wn  # noqa: E731
    _, ctx = _ctx([(0, n)], dtype=dtype)
    # all streams equal to one that is stored once
    stream = ResidualStream(x0.clone())
    _close(norm.forward_streams(stream, ctx, a.w_in, count), h(plain.gather_streams(streams, wa["in"])), dtype)
    assert stream.total.dim() == 2
    # the first update makes them differ, the second one acts on all of them at once
    stream = ResidualStream(stream.total, y1, links=a, stream_count=count)
    streams = plain.update_streams(streams, _cpu(y1), wa["mix"], wa["out"])
    _close(norm.forward_streams(stream, ctx, b.w_in, count), h(plain.gather_streams(streams, wb["in"])), dtype)
    assert stream.pending is None and stream.total.shape == (n, count, width)
    _close(stream.total, streams, torch.float32)
    stream = ResidualStream(stream.total, y2, links=b, stream_count=count)
    streams2 = plain.update_streams(streams, _cpu(y2), wb["mix"], wb["out"])
    # the norm ahead of the head: the sum of the streams, gathered rows, nothing written
    rows = torch.tensor([4, 0, 5], dtype=torch.int32, device=DEV)
    _close(norm.forward_streams(stream, ctx, None, count, rows=rows, num_rows=3, write=False), h(streams2.sum(1))[[4, 0, 5]], dtype)
    _close(stream.total, streams, torch.float32)
    _close(norm.forward_streams(stream, ctx, a.w_in, count), h(plain.gather_streams(streams2, wa["in"])), dtype)
    _close(stream.total, streams2, torch.float32)


def test_the_mix_matrix_is_indexed_from_to():
    """Stream 0 goes to stream 1 and nowhere else; a symmetric reading of the matrix would leave it where it is."""
    env = BuildEnv(torch.float32, DEV)
    norm = build_part("norm", PartSpec("rmsnorm", dict(size=8, eps=1e-6, name="g")), env)
    _bind(norm, torch.float32)
    links = StreamLinks(PartSpec("stream_links", dict(streams=2)), env)
    _bind(links, torch.float32, change=lambda t: (t["mix"].copy_(torch.tensor([[0.0, 1.0], [0.0, 0.0]])), t["out"].copy_(torch.tensor([0.0, 0.5]))))
    total = torch.stack((torch.full((1, 8), 3.0), torch.full((1, 8), 7.0)), dim=1).to(DEV)
    _, ctx = _ctx([(0, 1)])
    stream = ResidualStream(total.clone(), torch.full((1, 8), 10.0, device=DEV), links=links, stream_count=2)
    norm.forward_streams(stream, ctx, links.w_in, 2)
    assert stream.total[0, 0].tolist() == [0.0] * 8 and stream.total[0, 1].tolist() == [8.0] * 8


# --------------------------------------------------------------------------- attention
def _attention(dtype, heads, kv, dim, vdim, scale=0.3, v_mix=False):
    from miniserve_b200.models.tunadra import _attention as spec_of

    m = tx.attention_layer(heads, kv, dim, vdim, scale, v_mix)["mixer"]
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
@pytest.mark.parametrize("heads, kv, dim, vdim, page", [
    (6, 2, 16, 24, 16), (5, 1, 12, 20, 8), (4, 4, 20, 12, 8), (4, 2, 128, 128, 16), (8, 1, 96, 64, 16), (2, 1, 64, 128, 4), (1, 1, 8, 8, 16),
    (2, 1, 300, 40, 16), (16, 2, 48, 48, 32)])
def test_attention_whole_in_portions_and_decoded(dtype, heads, kv, dim, vdim, page):
    att, m = _attention(dtype, heads, kv, dim, vdim, scale=2.0 * dim ** -0.5)
    w = _bind(att, dtype)
    n = 61
    x = _x(n, dtype)
    x[7] *= 1e-3  # queries and keys far below one: the norm's eps shows
    ref = _attention_ref(x, w, m)
    full, ctx = _ctx([(0, n)], page, kv, att.cache_dim, dtype, seed=1)
    out = att.forward(x, ctx, KVEntryView(0, full.k_pool, full.v_pool, page))
    assert full.status.item() == 0
    _close(out, ref, dtype, 3.0)
    # what the cache holds: keys over their root mean square and the values as they are, zeros beyond their sizes
    k = full.read(0, full.k_pool, n).float().cpu()
    v = full.read(0, full.v_pool, n).float().cpu()
    _close(k[..., :dim], plain.rms((_cpu(x).double() @ w["k"].double().T).float().view(n, kv, dim), 1e-5), dtype, 2.0)
    _close(v[..., :vdim], (_cpu(x).double() @ w["v"].double().T).float().view(n, kv, vdim), dtype, 2.0)
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
    att, m = _attention(dtype, heads, kv, dim, 32, scale=24.0 / dim)
    w = _bind(att, dtype, change=lambda t: t["q"].copy_(
        t["k"].view(kv, 1, dim, HIDDEN).expand(kv, heads // kv, dim, HIDDEN).reshape(heads * dim, HIDDEN)))
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
@pytest.mark.parametrize("shapes", [((6, 2, 16, 24), (6, 3, 32, 16), (4, 1, 12, 48)), ((4, 2, 128, 128), (2, 1, 64, 256), (8, 8, 16, 32)),
                                    ((5, 5, 12, 4), (5, 1, 12, 20), (2, 2, 8, 10))])
def test_values_are_mixed_with_the_first_layers(dtype, shapes):
    """Three layers of one pass that share values, and one between that does not: what each caches, and its output. The layers split the same
    numbers into heads differently."""
    parts = [_attention(dtype, *s, scale=0.3, v_mix=True) for s in shapes]
    other, m_other = _attention(dtype, 2, 1, 16, 16)
    w_other = _bind(other, dtype, seed=9)
    ws = [_bind(p, dtype, seed=20 + i, change=lambda t, i=i: t["vmix"].fill_((0.7, 0.35, -0.25)[i])) for i, (p, _) in enumerate(parts)]
    n, page = 37, 8
    xs = [_x(n, dtype) for _ in parts]
    shared: dict = {}
    refs = [plain.attention(_cpu(x), w, "", m, 1e-5, torch.float32, shared) for x, w, (_, m) in zip(xs, ws, parts)]
    assert (refs[1] - plain.attention(_cpu(xs[1]), ws[1], "", parts[1][1], 1e-5, torch.float32)).abs().max() > 0.1  # the mixing shows
    pools = [_ctx([(0, n)], page, p.kv_heads, p.cache_dim, dtype, seed=30 + i)[0] for i, (p, _) in enumerate(parts)]
    other_pool, _ = _ctx([(0, n)], page, 1, 16, dtype, seed=40)
    for cuts in ((n,), (9, 2, 5, 2) + (1,) * n):  # whole, then portions and single tokens over the same pages
        at, outs = 0, [[] for _ in parts]
        for size in cuts:
            size = min(size, n - at)
            if size <= 0:
                break
            carried: dict = {}  # what the layers of one pass share
            bufs: dict = {}
            for i, (p, _) in enumerate(parts):
                _, ctx = _ctx([(at, size)], page, p.kv_heads, p.cache_dim, dtype, share=pools[i])
                ctx.buffers, ctx.step_cache = bufs, {k: v for k, v in carried.items() if k == "attn.v_first"}
                outs[i].append(p.forward(xs[i][at:at + size].contiguous(), ctx, KVEntryView(0, pools[i].k_pool, pools[i].v_pool, page)).clone())
                carried = ctx.step_cache
                if i == 0:
                    _, octx = _ctx([(at, size)], page, 1, 16, dtype, share=other_pool)
                    octx.buffers = bufs
                    other.forward(xs[1][at:at + size].contiguous(), octx, KVEntryView(0, other_pool.k_pool, other_pool.v_pool, page))
            at += size
        for i, (p, m) in enumerate(parts):
            _close(torch.cat(outs[i]), refs[i], dtype, 3.0)
            v = pools[i].read(0, pools[i].v_pool, n).float().cpu()[..., :m["vdim"]]
            own = (_cpu(xs[i]).double() @ ws[i]["v"].double().T).float()
            want = own if i == 0 else plain.mix_values(own, shared["v"], ws[i]["vmix"])
            _close(v.reshape(n, -1), want, dtype, 2.0)
    assert w_other["q"].shape[0] == 32


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_gate_per_head_reads_the_mixers_input(dtype):
    att, m = _attention(dtype, 4, 2, 16, 24)

    def gates(t):
        t["g"].zero_()
        t["g"][0, 0], t["g"][1, 0] = 40.0, -40.0  # channel 0 opens head 0 and shuts head 1
        t["o"].copy_(torch.cat((torch.eye(HIDDEN), torch.zeros(HIDDEN, 48)), dim=1))  # the first two heads' values come out as they are

    w = _bind(att, dtype, change=gates)
    x = _x(20, dtype)
    x[:, 0] = 1.0
    full, ctx = _ctx([(0, 20)], 8, 2, att.cache_dim, dtype)
    out = att.forward(x, ctx, KVEntryView(0, full.k_pool, full.v_pool, 8))
    _close(out, _attention_ref(x, w, m), dtype, 3.0)
    assert out[:, :24].abs().max() > 0.1 and out[:, 24:].abs().max() < 1e-6


# --------------------------------------------------------------------------- time mixing
def _time(dtype, heads, dim, rank):
    from miniserve_b200.models.tunadra import _wkv as spec_of

    m = dict(tx.wkv_layer(heads, dim)["mixer"], decay_rank=rank)
    return build_part("mixer", spec_of(HIDDEN, 1e-5, m), BuildEnv(dtype, DEV)), m


def _time_weights(t):
    c = t["w0"].numel()
    t["w0"].copy_(torch.linspace(-5.5, 1.5, c)[torch.randperm(c, generator=torch.Generator().manual_seed(5))])
    for x in "rkvgw":
        t["mu." + x].copy_(torch.linspace(-0.2, 1.2, HIDDEN)[torch.randperm(HIDDEN, generator=torch.Generator().manual_seed(ord(x)))])
    t["u"].mul_(3.0)


def _views(part, slots=5):
    """Slots that hold NaN: nothing of it may show in a sequence that starts there."""
    return tuple(StateEntryView(torch.full((slots, *nd.shape), float("nan"), dtype=nd.dtype, device=DEV), tuple(nd.shape)) for nd in part.cache_need())


def _portions(part, views, x, cuts, slot, dtype):
    outs, at = [], 0
    for size in cuts:
        size = min(size, x.shape[0] - at)
        if size <= 0:
            break
        _, ctx = _ctx([(at, size)], dtype=dtype, slots=[slot])
        outs.append(part.forward(x[at:at + size].contiguous(), ctx, views).clone())
        at += size
    return torch.cat(outs)


def _time_ref(x, w, m, dtype):
    ref = plain.wkv(_cpu(x), w, "", m, 1e-5, torch.float32, acc=torch.float64)
    noise = (plain.wkv(_cpu(x), w, "", m, 1e-5, dtype) - ref).abs().amax(dim=1)
    return ref, noise


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, dim, rank", [(3, 16, 12), (5, 24, 7), (3, 10, 5), (1, 6, 1), (2, 20, 16), (3, 64, 32), (2, 128, 24), (1, 8, 3), (2, 72, 64), (1, 200, 8)])
def test_time_mixing_whole_in_portions_and_decoded(dtype, heads, dim, rank):
    part, m = _time(dtype, heads, dim, rank)
    w = _bind(part, dtype, change=_time_weights)
    n = 150
    x = _x(n, dtype)
    ref, noise = _time_ref(x, w, m, dtype)
    views = _views(part)
    _close(_portions(part, views, x, (n,), 1, dtype), ref, dtype, 3.0, noise)
    # the same slot again; single tokens from the very first one, portions down to two tokens, a chunk and one token less and more, then token by token
    _close(_portions(part, views, x, (1, 1, 2, 1, 3, 2, 17, 2, 9, 64, 2) + (1,) * n, 1, dtype), ref, dtype, 3.0, noise)
    _close(_portions(part, views, x, (63, 65, 2) + (1,) * n, 2, dtype), ref, dtype, 3.0, noise)
    _, ctx = _ctx([(0, 71), (0, n - 9)], dtype=dtype, slots=[4, 0])
    both = part.forward(torch.cat((x[:71], x[:n - 9])), ctx, views)
    _close(both, torch.cat((ref[:71], ref[:n - 9])), dtype, 3.0, torch.cat((noise[:71], noise[:n - 9])))
    _, ctx = _ctx([(n - 9, 1), (71, 70)], dtype=dtype, slots=[0, 4])
    both = part.forward(torch.cat((x[n - 9:n - 8], x[71:141])), ctx, views)
    _close(both, torch.cat((ref[n - 9:n - 8], ref[71:141])), dtype, 3.0, torch.cat((noise[n - 9:n - 8], noise[71:141])))
    _, ctx = _ctx([(n - 8, 1), (0, 1), (141, 1)], dtype=dtype, slots=[0, 3, 4])  # three decoding rows, one of them at its very first token
    rows = part.forward(torch.cat((x[n - 8:n - 7], x[:1], x[141:142])), ctx, views)
    pick = [n - 8, 0, 141]
    _close(rows, ref[pick], dtype, 3.0, noise[pick])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, dim", [(2, 24), (2, 64), (1, 128), (3, 12)])
def test_time_mixing_over_a_long_portion_and_long_decoding(dtype, heads, dim):
    """Portions of hundreds of tokens (chunks, or a walk in segments), behind an earlier portion, beside a short row, and hundreds of
    tokens decoded one by one from the state they left."""
    part, m = _time(dtype, heads, dim, 16)
    w = _bind(part, dtype, change=_time_weights)
    n = 1000
    x = _x(n, dtype)
    ref, noise = _time_ref(x, w, m, dtype)
    views = _views(part)
    _close(_portions(part, views, x[:700], (700,), 1, dtype), ref[:700], dtype, 3.0, noise[:700])
    _close(_portions(part, views, x, (37, 663) + (1,) * n, 2, dtype), ref, dtype, 3.0, noise)
    _, ctx = _ctx([(0, 5), (0, 690)], dtype=dtype, slots=[4, 0])
    both = part.forward(torch.cat((x[:5], x[:690])), ctx, views)
    _close(both, torch.cat((ref[:5], ref[:690])), dtype, 3.0, torch.cat((noise[:5], noise[:690])))


def _walk(r, k, v, decay, u, start):
    """The recurrence in 64-bit: r, k, decay [n, H, d], v [n, H, e], start [H, e, d] -> outputs [n, H, e], their sizes, last state."""
    s, outs, sizes = start.clone(), [], []
    for i in range(r.shape[0]):
        kv = v[i][:, :, None] * k[i][:, None, :]
        seen = s + u[:, None, :] * kv
        outs.append((seen * r[i][:, None, :]).sum(-1))
        sizes.append((seen.abs() * r[i].abs()[:, None, :]).sum(-1) + 1e-3)
        s = decay[i][:, None, :] * s + kv
    return torch.stack(outs), torch.stack(sizes), s


BONUS_ROWS = [(0, 1), (5, 64), (0, 65), (300, 200), (0, 7), (9, 1), (0, 129), (64, 16), (0, 48)]


def _bonus_case(heads, d, e, dtype, seed=0):
    gen = torch.Generator().manual_seed(seed)
    t = sum(n for _, n in BONUS_ROWS)
    r, k, v = (torch.randn(t, heads * n, generator=gen).to(torch.bfloat16).to(dtype).to(DEV) for n in (d, d, e))
    z = torch.rand(t, heads * d, generator=gen) * 9.0 - 7.0
    z[::17] = 30.0        # a decay of exactly zero
    z[5::29] = -40.0      # of exactly one
    z[70:90] = 4.0        # of about 1e-24, for several tokens in a row
    w0, u = torch.randn(heads * d, generator=gen) * 0.3, torch.randn(heads * d, generator=gen) * 2
    state = torch.randn(len(BONUS_ROWS), heads, e, d, generator=gen)
    return t, r, k, v, z.to(DEV), w0.to(DEV), u.to(DEV), state.to(DEV)


def _bonus_check(o, state, held, r, k, v, z, w0, u, ctx, heads, d, e, tol):
    rd, kd, vd = (x.double().cpu().view(x.shape[0], heads, -1) for x in (r, k, v))
    decay = torch.exp(-torch.exp(z.double().cpu() + w0.double().cpu())).view(z.shape[0], heads, d)
    at = 0
    for (start, n), slot in zip(BONUS_ROWS, ctx.state_slot.tolist()):
        s0 = held[slot].double().cpu() if start else torch.zeros(heads, e, d, dtype=torch.float64)
        want, size, last = _walk(rd[at:at + n], kd[at:at + n], vd[at:at + n], decay[at:at + n], u.double().cpu().view(heads, d), s0)
        err = ((o[at:at + n].double().cpu() - want).abs() / size).amax(dim=(1, 2))
        assert err.max() < tol, (slot, int(err.argmax()), err.max().item())
        assert (state[slot].double().cpu() - last).abs().max() < tol * max(1.0, last.abs().max().item())
        at += n


@pytest.mark.parametrize("heads, d, e", [(2, 64, 64), (3, 16, 24), (1, 128, 128), (2, 40, 72), (1, 8, 8), (2, 96, 160)])
def test_bonus_rule_over_chunks_on_the_tensor_cores(heads, d, e):
    """Rows from one token to several chunks, some behind an earlier state, decays of zero, of one and of next to nothing, against the recurrence
    in 64-bit: the tensor cores see what is not exact in bfloat16 as two numbers, so the error stays far below bfloat16's."""
    _, ctx = _ctx(BONUS_ROWS, dtype=torch.bfloat16, slots=[6, 0, 3, 1, 4, 5, 2, 8, 7])
    t, r, k, v, z, w0, u, state = _bonus_case(heads, d, e, torch.bfloat16)
    held = state.clone()
    o = torch.full((t, heads, e), float("nan"), device=DEV)
    assert ops.time_chunks_ok(r, k, v, d, e, ctx)
    ops.time_chunks(o, state, r, k, v, z, w0, u, ctx, heads, d, e, None, None, 1e-5, raw=True)
    _bonus_check(o, state, held, r, k, v, z, w0, u, ctx, heads, d, e, 6e-5)
    # with the norm and the gate behind it (inside the kernel for heads of up to 64 values)
    gate, norm_w = torch.randn(t, heads * e, device=DEV).bfloat16(), torch.randn(heads * e, device=DEV)
    out = torch.full((t, heads * e), float("nan"), device=DEV, dtype=torch.bfloat16)
    state = held.clone()
    ops.time_chunks(out, state, r, k, v, z, w0, u, ctx, heads, d, e, gate, norm_w, 1e-5)
    want = plain.rms(o.cpu(), 1e-5).reshape(t, -1) * norm_w.cpu() * plain.silu(gate.float().cpu())
    assert ((out.float().cpu() - want).abs() <= 5e-3 * want.abs() + 1e-3).all()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, d, e", [(2, 64, 64), (3, 16, 24), (1, 10, 6), (1, 300, 40)])
def test_bonus_rule_token_by_token(dtype, heads, d, e):
    """The walk (rows in one piece, and cut into segments: the step has more than 512 tokens), same cases."""
    t, r, k, v, z, w0, u, state = _bonus_case(heads, d, e, dtype, seed=1)
    for segments in (1, 8):
        _, ctx = _ctx(BONUS_ROWS, dtype=dtype, slots=[6, 0, 3, 1, 4, 5, 2, 8, 7])
        decay = torch.empty_like(z)
        ops.channel_decay(decay, z, w0)
        st = state.clone()
        o = torch.full((t, heads, e), float("nan"), device=DEV)
        from miniserve_b200.ops import mixers

        held, mixers.SEGMENTS = mixers.SEGMENTS, segments
        try:
            ops.decay_scan(o, st, r, k, v, decay, None, None, 0.0, None, ctx, heads, d, e, 1.0, delta=False, bonus=u)
        finally:
            mixers.SEGMENTS = held
        _bonus_check(o, st, state, r, k, v, z, w0, u, ctx, heads, d, e, 2e-5)


@pytest.mark.parametrize("dtype", DTYPES)
def test_the_bonus_is_the_current_tokens_alone(dtype):
    """One head whose channels forget everything at once: an output is the token's own k v^T times the bonus plus the token before's as it was
    written; without the bonus half of it is missing, and a read-out behind the write would count the token twice."""
    part, m = _time(dtype, 1, 16, 4)

    def forget(t):
        t["w1"].zero_()
        t["w0"].fill_(5.0)  # exp(-exp(5)) is zero
        t["u"].fill_(2.0)
        for x in "rkvgw":
            t["mu." + x].zero_()

    w = _bind(part, dtype, change=forget)
    n = 80
    x = _x(n, dtype)
    ref, noise = _time_ref(x, w, m, dtype)
    h = _cpu(x)
    r, k, v, g = ((h @ w[q].T) for q in "rkvg")
    o = 2.0 * (r * k).sum(-1, keepdim=True) * v
    o[1:] += (r[1:] * k[:-1]).sum(-1, keepdim=True) * v[:-1]
    want = (plain.rms(o, 1e-5) * w["norm"] * plain.silu(g)) @ w["o"].T
    assert (want - ref).abs().max() < 1e-3 * want.abs().max()
    views = _views(part)
    _close(_portions(part, views, x, (n,), 0, dtype), ref, dtype, 3.0, noise)
    _close(_portions(part, views, x, (2,) * 10 + (1,) * n, 0, dtype), ref, dtype, 3.0, noise)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dim", [16, 64, 10])
def test_time_mixing_keeps_an_early_token_in_slow_channels(dtype, dim):
    """Head 0 hardly forgets and head 1 forgets within a few tokens: a change of the first tokens must show in the last one's features through
    head 0, decoded and in a prompt, and not through head 1."""
    part, m = _time(dtype, 2, dim, 4)

    def decays(t):
        t["w1"].zero_()
        t["w0"].copy_(torch.cat((torch.full((dim,), -9.0), torch.full((dim,), 1.0))))

    w = _bind(part, dtype, change=decays)
    n = 140
    x = _x(n, dtype)
    other = x.clone()
    other[:3] = _x(3, dtype, 6.0)
    views = _views(part)
    feats = []
    for inp in (x, other):
        for cuts in ((n - 1, 1), (70, n - 70)):
            at = 0
            for size in cuts:
                _, ctx = _ctx([(at, size)], dtype=dtype, slots=[3])
                f = torch.zeros(size, part.feature_width, device=DEV, dtype=dtype)
                part.features(inp[at:at + size].contiguous(), ctx, views, f)
                at += size
            feats.append(f.float().cpu()[-1])
    for a, b in ((feats[0], feats[2]), (feats[1], feats[3])):
        diff = (a - b).abs()
        assert diff[:dim].max() > 5e-2 and diff[dim:].max() < 1e-3
    ref, noise = _time_ref(other, w, m, dtype)
    _close(_portions(part, views, other, (n,), 0, dtype), ref, dtype, 3.0, noise)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [40, 36, 1024, 2056])
def test_token_mixes_and_the_state_they_leave(dtype, width):
    mix = torch.rand(5, width, device=DEV) * 2 - 0.5
    h = torch.randn(1500, width, device=DEV).to(dtype)
    want = torch.stack([plain.shift_mix(_cpu(h), mix[m].cpu()) for m in range(5)])
    state = torch.full((3, width), float("nan"), dtype=dtype, device=DEV)

    def run(rows, slots, x):
        _, ctx = _ctx(rows, dtype=dtype, slots=slots)
        out = torch.empty(5, x.shape[0], width, dtype=dtype, device=DEV)
        ops.token_mixes(out, x, state, mix, ctx)
        return out

    def close(got, ref):
        assert (got.float().cpu() - ref).abs().max() < (1e-5 if dtype == torch.float32 else 4e-2)

    close(run([(0, 1500)], [1], h), want)
    assert torch.equal(state[1], h[-1])
    at = 0
    for n in (1, 1, 2, 1200, 3, 1, 292):
        close(run([(at, n)], [2], h[at:at + n].contiguous()), want[:, at:at + n])
        at += n
    close(run([(700, 1), (0, 1101), (0, 2)], [0, 1, 2], torch.cat((h[700:701], h[:1101], h[:2])))[:, 1:], torch.cat((want[:, :1101], want[:, :2]), dim=1))
    assert torch.equal(state[0], h[700]) and torch.equal(state[1], h[1100]) and torch.equal(state[2], h[1])


@pytest.mark.parametrize("m", [1, 5, 8, 9, 16])
@pytest.mark.parametrize("c, rank, k", [(48, 16, 64), (1024, 64, 1024), (160, 8, 72)])
def test_one_launch_for_the_products_of_several_inputs(m, c, rank, k):
    x = torch.randn(5, m, k, device=DEV).bfloat16()
    w = (torch.randn(4 * c + rank, k, device=DEV) * k ** -0.5).bfloat16()
    assert ops.linear_inputs_ok(x, w, c) and not ops.linear_inputs_ok(x, w, c + 8)
    out = ops.linear_inputs(x, w, torch.empty(m, 4 * c + rank, device=DEV, dtype=torch.bfloat16), c, 4 * c)
    want = torch.cat([x[i].float() @ w[i * c:(i + 1) * c].float().T for i in range(4)] + [torch.tanh(x[4].float() @ w[4 * c:].float().T)], dim=1)
    assert (out.float() - want).abs().max() < 2e-2


# --------------------------------------------------------------------------- feed-forward
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("hidden, ff, experts, top, count, keep, shared", [
    (48, 24, 6, 2, 3, 2, 40), (36, 20, 5, 1, 0, 0, 28), (40, 12, 1, 1, 0, 0, 0), (64, 64, 8, 4, 2, 1, 96), (56, 24, 4, 3, 4, 3, 0), (128, 136, 32, 8, 4, 2, 72),
    (48, 20, 12, 6, 3, 3, 44), (64, 32, 96, 40, 8, 7, 0)])
def test_router_and_experts(dtype, hidden, ff, experts, top, count, keep, shared):
    from miniserve_b200.models.tunadra import _feed_forward as spec_of

    mlp = tx.moe(ff, experts, top, count, keep, scale=1.7, limit=0.9, shared=shared, shared_limit=0.4)
    ffn = build_part("feed_forward", spec_of(hidden, mlp), BuildEnv(dtype, DEV))
    w = _bind(ffn, dtype, change=lambda t: t["router"].mul_(1.5))
    for n in (1, 2, 77, 600):
        x = torch.randn(n, hidden, device=DEV).to(dtype)
        _, ctx = _ctx([(0, n)], dtype=dtype)
        idx, wgt = ffn.route(x, ctx)
        chosen, weights = plain.route(_cpu(x), w, "", mlp["router"], torch.float32)
        order_g, order_w = idx.long().cpu().sort(-1), chosen.sort(-1)
        assert (order_g.values == order_w.values).all()
        assert torch.allclose(wgt.cpu().gather(1, order_g.indices), weights.gather(1, order_w.indices), rtol=1e-4, atol=1e-6)
        assert torch.allclose(wgt.sum(-1).cpu(), torch.full((n,), 1.7), rtol=1e-4)
        want = plain.moe_ff(_cpu(x), w, "", mlp, torch.float32)
        _close(ffn.forward(x, ctx), want, dtype, 3.0)
        if dtype == torch.bfloat16:
            held = xo.TC_EXPERTS  # the products on the older tensor-core path too (what shapes off the tcgen05 kernel's take)
            xo.TC_EXPERTS = False
            try:
                _close(ffn.forward(x, ctx), want, dtype, 3.0)
            finally:
                xo.TC_EXPERTS = held
            for config in (1, 2):  # both tilings of the grouped products
                native.gemm_tc().ms_gemm_tc_set_grouped(config)
                try:
                    _close(ffn.forward(x, ctx), want, dtype, 3.0)
                finally:
                    native.gemm_tc().ms_gemm_tc_set_grouped(0)


def _route(scores, router, dtype=torch.float32, correction=None, **kw):
    """The engine's choice where the router's scores are given (one token, input one)."""
    w = torch.tensor([[math.log(p / (1 - p))] for p in scores], device=DEV)
    w = torch.cat((w, torch.zeros(len(scores), 3, device=DEV)), dim=1).contiguous()
    x = torch.zeros(1, 4, device=DEV, dtype=dtype)
    x[0, 0] = 1.0
    idx, wgt = torch.empty(1, router["top"], dtype=torch.int32, device=DEV), torch.empty(1, router["top"], device=DEV)
    g = router.get("groups") or {"count": 1, "keep": 1}
    xo.expert_route(idx, wgt, x, w, correction, router["top"], g["count"], g["keep"], router.get("scale", 1.0), True, score="sigmoid", **kw)
    return idx[0].tolist(), wgt[0].cpu()


def test_groups_are_chosen_by_their_two_largest_scores():
    scores = [0.99, 0.02, 0.01, 0.03] + [0.7, 0.6, 0.1, 0.1] + [0.65, 0.1, 0.2, 0.55]
    router = {"top": 3, "groups": {"count": 3, "keep": 2}, "scale": 2.0}
    idx, wgt = _route(scores, router, group_best=2, renorm_eps=1e-20)
    assert idx == [4, 8, 5] and torch.allclose(wgt, 2.0 * torch.tensor([0.7, 0.65, 0.6]) / 1.95, rtol=1e-5)
    assert _route(scores, router, group_best=1)[0] == [0, 4, 5]  # by the largest alone the first group would have been kept
    # equal scores inside a group count twice: 0.5 + 0.5 beats 0.8 + 0.1
    assert _route([0.8, 0.1, 0.05] + [0.5, 0.5, 0.05] + [0.01, 0.02, 0.03], {"top": 2, "groups": {"count": 3, "keep": 1}}, group_best=2)[0] == [3, 4]
    # three of a group
    assert _route([0.8, 0.1, 0.05] + [0.4, 0.3, 0.28] + [0.01, 0.02, 0.03], {"top": 2, "groups": {"count": 3, "keep": 1}}, group_best=3)[0] == [3, 4]


@pytest.mark.parametrize("dtype", DTYPES)
def test_limits_of_the_experts_and_of_the_shared_one(dtype):
    """Gates and ups far beyond both limits: an expert's inner values are the limits' alone, with the shared expert's own."""
    from miniserve_b200.models.tunadra import _feed_forward as spec_of

    mlp = tx.moe(24, 4, 1, 0, 0, scale=1.0, limit=2.0, shared=40, shared_limit=0.5)
    ffn = build_part("feed_forward", spec_of(HIDDEN, mlp), BuildEnv(dtype, DEV))

    def far(t):
        for k in t:
            if k.endswith((".gate", ".up")):
                t[k].zero_()
                t[k][:, 0] = 30.0
            elif k.endswith(".down"):
                t[k].fill_(0.25)

    w = _bind(ffn, dtype, change=far)
    inner = lambda c: c / (1 + math.exp(-1.702 * c)) * (c + 1)  # noqa: E731
    for n in (2, 40):  # a decode step's products, a prompt's
        x = _x(n, dtype)
        x[:, 0] = 1.0
        _, ctx = _ctx([(0, n)], dtype=dtype)
        out = ffn.forward(x, ctx)
        _close(out, plain.moe_ff(_cpu(x), w, "", mlp, torch.float32), dtype, 3.0)
        want = 0.25 * (24 * inner(2.0) + 40 * inner(0.5))
        assert (out.float() - want).abs().max() < 0.02 * want


# --------------------------------------------------------------------------- whole models
@pytest.fixture(scope="module", params=["a", "b", "c", "d"])
def model(request, tmp_path_factory):
    raw = getattr(tx, "config_" + request.param)()
    folder = tx.write_model(tmp_path_factory.mktemp("tunadra_" + request.param), raw, seed=ord(request.param))
    return dict(folder=folder, raw=raw, oracle=tx.oracle(folder), rounded=tx.oracle(folder, torch.bfloat16),
                page=dict(a=16, b=8, c=32, d=16)[request.param])


def _logits_close(model, dtype, got, ids, what=""):
    """32-bit: within F32 of the oracle. bfloat16: as near as rounding allows, position by position (``tx.rounded_ok``)."""
    want = model["oracle"](ids)
    if dtype == "float32":
        ok, report = tx.float32_ok(model["folder"], got, want, ids, F32)
        assert ok, f"{what}: {report}"
    else:
        ok, report = tx.rounded_ok(got, want, model["rounded"](ids))
        assert ok, f"{what}: {report}"


def test_layer_streams_in_float32(model):
    """The sum of the residual streams after every layer, against the oracle's."""
    from miniserve_b200.cache import CacheManager
    from miniserve_b200.engine.loader import load_model
    from miniserve_b200.engine.step import StepFunction, StepRow

    ids = _ids(29, model["raw"]["vocab"], 8)
    want = tx.layer_streams(model["folder"], ids)
    _, _, net = load_model(model["folder"], "float32", "cuda:0")
    cache = CacheManager(net.entry_caches, 8, 16, 2, dtype=net.dtype, device=net.device)
    ctx = StepFunction(net, cache).prepare([StepRow(cache.new_request(), ids, [0])])
    stream = ResidualStream(net.embed(ctx, cache.entry_views))
    count = model["raw"]["streams"]
    for i, e in enumerate(net.spec.run_order):
        stream = net.layers[e.layer].forward(stream, ctx, cache.entry_views[i])
        total = _cpu(stream.total) if stream.total.dim() == 3 else _cpu(stream.total)[:, None, :].repeat(1, count, 1)
        x = plain.update_streams(total, _cpu(stream.pending), stream.links.w_mix.cpu(), stream.links.w_out.cpu()).sum(1)
        assert (x - want[i]).abs().max() < 1e-4 * max(1.0, want[i].abs().max().item()), f"after layer {i}"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_whole_decoded_and_in_portions(model, dtype):
    vocab = model["raw"]["vocab"]
    run = tx.Runner(model["folder"], dtype, max_tokens=256, page_size=model["page"])
    for n, seed in ((1, 1), (2, 2), (37, 3), (170, 4)):
        ids = _ids(n, vocab, seed)
        _logits_close(model, dtype, run.feed("w", ids, [n]), ids, f"{n} whole")
        if n > 2:
            _logits_close(model, dtype, run.feed("d", ids, [n - min(n - 1, 110), 1]), ids, f"{n} decoded")
            _logits_close(model, dtype, run.feed("c", ids, [7, 2, 24, 3, model["page"], 2, 65, 31, 2, 1, 1, 2, 9]), ids, f"{n} in portions")
        assert run.cache.is_idle()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_mixed_batches_reuse_pages_and_slots(model, dtype):
    """Up to four live requests, portions of some beside single tokens of others, a pool that holds only what is live and
    four state slots: every page and slot is used by several requests in turn (pages are filled with NaN when given back)."""
    vocab = model["raw"]["vocab"]
    seqs = {f"r{i}": _ids(n, vocab, 20 + i) for i, n in enumerate([90, 5, 64, 33, 1, 120, 17, 48, 2, 75])}
    run = tx.Runner(model["folder"], dtype, max_tokens=4 * 128, page_size=model["page"], max_requests=4)
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
    run = tx.Runner(model["folder"], "float32", max_tokens=448, page_size=model["page"])
    _logits_close(model, "float32", run.feed("long", ids, [3, 1]), ids)


def test_a_long_prompt_whole_and_in_two_portions(model):
    ids = _ids(1200, model["raw"]["vocab"], 10)
    run = tx.Runner(model["folder"], "float32", max_tokens=1216, page_size=model["page"])
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
            slack = 1e-3 if dtype == "float32" else max(0.15, 3.0 * moved[at].item())
            assert (logits.max() - logits[t]).item() <= slack, (at + 1, t)


def test_recurring_prompt_steps_replay_from_graphs(model):
    """The same prompts again and again: their steps are captured and replayed, and the tokens stay the same."""
    from miniserve_b200.engine import LLM, SamplingParams

    vocab = model["raw"]["vocab"]
    llm = LLM(model["folder"], dtype="bfloat16", kv_pool_tokens=1024, page_size=model["page"], max_running=2, chunked_prefill_size=128)
    prompts = [_ids(90, vocab, 50), _ids(33, vocab, 51)]
    first = [llm.generate([p], SamplingParams(max_new_tokens=4))[0] for p in prompts]
    for _ in range(12):
        for p, want in zip(prompts, first):
            assert llm.generate([p], SamplingParams(max_new_tokens=4))[0] == want
    assert llm.engine.cache.is_idle()


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
            assert (logits.max() - logits[t]).item() <= 1e-3
