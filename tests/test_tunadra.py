"""Tunadra without a GPU: configuration -> parts and run order, declared tensors against a statement of the
checkpoint format, cache needs, refused configurations, and the oracle's functions against other statements
of the same formulas."""

import json
import math

import pytest
import torch

from miniserve_b200.cache.manager import CacheManager, group_needs
from miniserve_b200.config import preset
from miniserve_b200.config.registry import resolve
from miniserve_b200.parts import FixedState, PagedKV
from miniserve_b200.parts.decoder import DecoderModel
from tests import tunadra_util as tx
from tests.plain import tunadra_plain as plain


# --------------------------------------------------------------------------- configuration
@pytest.mark.parametrize("make", [tx.config_a, tx.config_b, tx.config_c, tx.config_d])
def test_declared_tensors_are_the_checkpoint_format(make):
    raw = make()
    _, _, spec = resolve(tx.resolved(raw))
    model = DecoderModel(spec, torch.bfloat16, "cpu")
    decls = model.weight_decls()
    assert {k: tuple(v.shape) for k, v in decls.items()} == tx.tensor_shapes(raw)
    assert spec.vocab_size == raw["vocab"] and spec.hidden_size == raw["width"] and model.shape_static
    # what mixes the streams, enters the recurrence besides the products, and chooses experts stays in 32-bit
    kept = {k for k, v in decls.items() if v.precision == "float32"}
    assert kept == {k for k in decls if ".hc" in k or ".mu." in k or k.rsplit(".", 1)[-1] in ("w0", "u", "router", "vmix") or k.endswith("mix.norm")}


def test_the_decays_rank_is_read_off_the_checkpoint(tmp_path):
    raw = tx.config_a()
    folder = tx.write_model(tmp_path / "m", raw, seed=1)
    plain_raw = json.loads((folder / "config.json").read_text())
    with pytest.raises(KeyError):
        resolve(plain_raw)
    _, cfg, spec = resolve(plain_raw, folder)
    assert [layer.mixer["decay_rank"] for layer in cfg.layers if layer.type == "wkv"] == [12, 7]
    assert "decay_rank" not in plain_raw["layers"][0]["mixer"]


def test_cache_needs_follow_the_mixers():
    _, _, spec = resolve(tx.resolved(tx.config_a()))
    model = DecoderModel(spec, torch.bfloat16, "cpu")
    needs = [c.need for c in model.entry_caches]
    f32, bf = torch.float32, torch.bfloat16
    assert needs[0] == (FixedState((3, 16, 16), f32), FixedState((64,), bf))  # S of every head, the last input
    assert needs[1] == PagedKV(2, 32, None) and needs[2] == PagedKV(4, 32, None)  # keys and values in heads of whole sixteens
    assert needs[3] == (FixedState((5, 24, 24), f32), FixedState((64,), bf))
    groups, states = group_needs(model.entry_caches)
    assert len(states) == 4
    cache = CacheManager(model.entry_caches, 4, 16, 2, device=None)
    rc = cache.new_request()
    cache.reserve([(rc, 33)])
    assert set(cache.num_free()) == {1}
    cache.release(rc)
    assert cache.is_idle()


def test_a_model_without_attention_has_no_pages():
    _, _, spec = resolve(tx.resolved(tx.config_d()))
    model = DecoderModel(spec, torch.bfloat16, "cpu")
    cache = CacheManager(model.entry_caches, 4, 16, 2, device=None)
    rc = cache.new_request()
    cache.reserve([(rc, 1000)])
    assert cache.num_groups == 0 and rc.num_tokens == 1000


@pytest.mark.parametrize("change, error", [
    (lambda r: r["layers"][0].update(type="mamba2"), NotImplementedError),
    (lambda r: r["layers"][0]["mlp"].update(kind="dense"), NotImplementedError),
    (lambda r: r["layers"][0]["mixer"].pop("decay_rank"), KeyError),
    (lambda r: r["layers"][0]["mixer"].update(heads=0), ValueError),
    (lambda r: r["layers"][1]["mixer"].update(kv_heads=4), ValueError),
    (lambda r: r["layers"][4]["mixer"].update(vdim=24), ValueError),
    (lambda r: r["layers"][1]["mlp"]["router"].update(top=7), ValueError),
    (lambda r: r["layers"][1]["mlp"]["router"]["groups"].update(count=4), ValueError),
    (lambda r: r["layers"][1]["mlp"]["router"]["groups"].update(keep=1), ValueError),
    (lambda r: r["layers"][1]["mlp"]["shared"].update(limit=-1.0), ValueError),
    (lambda r: r.update(streams=0), ValueError),
    (lambda r: r.update(logit_softcap=0.0), ValueError),
    (lambda r: r.update(layers=[]), ValueError),
    (lambda r: r.pop("streams"), KeyError),
])
def test_refused_configurations(change, error):
    raw = tx.resolved(tx.config_a())
    change(raw)
    with pytest.raises(error):
        resolve(raw)


def test_the_preset_and_optional_tensors():
    _, _, spec = resolve(preset("tunadra-tiny"))
    assert [layer.mixer.kind for layer in spec.layers] == ["time_mix", "gqa_attention", "time_mix", "gqa_attention"]
    _, _, spec_a = resolve(tx.resolved(tx.config_a()))
    # the layer without a feed-forward, which also shares no values
    assert set(spec_a.optional_tensors) == {"l2.norm2", "l2.hc2.in", "l2.hc2.out", "l2.hc2.mix", "l2.mix.vmix"}
    assert spec_a.layers[0].feed_forward["shared_glu"] == {"limit": 0.8} and spec_a.layers[0].feed_forward["limit"] == 1.5


# --------------------------------------------------------------------------- the oracle against other statements
def test_streams_are_matrices():
    torch.manual_seed(0)
    x, y = torch.randn(5, 3, 7), torch.randn(5, 7)
    mix, out, into = torch.randn(3, 3), torch.randn(3), torch.randn(3)
    want = torch.einsum("nsw,st->ntw", x, mix) + out[None, :, None] * y[:, None, :]
    assert torch.allclose(plain.update_streams(x, y, mix, out), want, atol=1e-5)
    assert torch.allclose(plain.gather_streams(x, into), torch.einsum("nsw,s->nw", x, into), atol=1e-5)


def test_time_mixing_equals_its_quadratic_form():
    """o_i = sum over j < i of (sum_c r_i k_j times the decays between) v_j, and the token's own k v^T times the bonus."""
    torch.manual_seed(1)
    t, h, d, e = 12, 2, 4, 5
    r, k, v = (torch.randn(t, h, n, dtype=torch.float64) for n in (d, d, e))
    decay, u = torch.rand(t, h, d, dtype=torch.float64), torch.randn(h, d, dtype=torch.float64)
    got = plain.bonus_scan(r, k, v, decay, u)
    for hd in range(h):
        for i in range(t):
            want = (r[i, hd] * u[hd] * k[i, hd]).sum() * v[i, hd]
            for j in range(i):
                between = decay[j + 1:i, hd].prod(dim=0)  # the tokens between j and i: neither's own
                want = want + (r[i, hd] * between * k[j, hd]).sum() * v[j, hd]
            assert (got[i, hd] - want).abs().max() < 1e-10


def test_decay_shift_and_value_mixing():
    z = torch.tensor([-20.0, 0.0, 1.0, 30.0])
    assert torch.allclose(plain.channel_decay(z), torch.tensor([math.exp(-math.exp(-20.0)), math.exp(-1.0), math.exp(-math.e), 0.0]))
    h = torch.tensor([[1.0, 2.0], [5.0, 6.0], [0.0, -1.0]])
    assert torch.equal(plain.shift_mix(h, torch.tensor([1.0, 0.0])), torch.tensor([[0.0, 2.0], [1.0, 6.0], [5.0, -1.0]]))
    assert torch.allclose(plain.mix_values(torch.tensor([4.0]), torch.tensor([8.0]), torch.tensor(0.25)), torch.tensor([5.0]))


def test_router_keeps_the_groups_with_the_largest_two():
    """One expert of score 0.99 beside three low ones loses to a group of two middling ones."""
    logit = lambda p: math.log(p / (1 - p))  # noqa: E731
    scores = [0.99, 0.02, 0.01, 0.03] + [0.7, 0.6, 0.1, 0.1] + [0.65, 0.1, 0.2, 0.55]
    w = {"router": torch.tensor([[logit(p)] for p in scores])}
    router = {"experts": 12, "top": 3, "groups": {"count": 3, "keep": 2}, "scale": 2.0}
    chosen, weights = plain.route(torch.ones(1, 1), w, "", router, torch.float32)
    assert sorted(chosen[0].tolist()) == [4, 5, 8]
    assert abs(weights.sum().item() - 2.0) < 1e-5 and abs(weights[0].max().item() - 2.0 * 0.7 / 1.95) < 1e-4
    router["groups"]["keep"] = 3
    assert 0 in plain.route(torch.ones(1, 1), w, "", router, torch.float32)[0][0].tolist()


def test_clamped_glu_and_softcap():
    g, u = torch.tensor([9.0, -9.0, 0.5]), torch.tensor([9.0, -9.0, 0.5])
    sig = lambda x: 1 / (1 + math.exp(-x))  # noqa: E731
    want = [2 * sig(3.404) * 3.0, -9 * sig(-15.318) * -1.0, 0.5 * sig(0.851) * 1.5]
    assert torch.allclose(plain.clamped_glu(g, u, 2.0), torch.tensor(want), atol=1e-6)
    assert torch.allclose(plain.softcap(torch.tensor([0.1, 1000.0]), 5.0), torch.tensor([5 * math.tanh(0.02), 5.0]))


def test_sinusoid():
    s = plain.sinusoid(torch.arange(40), 6)
    for p in (0, 1, 39):
        for i in range(3):
            ang = p * 10000.0 ** (-2.0 * i / 6)
            assert abs(s[p, 2 * i] - math.sin(ang)) < 1e-5 and abs(s[p, 2 * i + 1] - math.cos(ang)) < 1e-5
