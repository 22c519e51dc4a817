"""Vumedra without a GPU: configuration -> parts and run order, declared tensors against a statement of the
checkpoint format, cache needs, refused configurations, and the oracle's functions against other statements
of the same formulas."""

import math

import numpy as np
import pytest
import torch

from miniserve_b200.cache.manager import CacheManager, group_needs
from miniserve_b200.config import preset
from miniserve_b200.config.registry import resolve
from miniserve_b200.parts import FixedState, PagedKV
from miniserve_b200.parts.decoder import DecoderModel
from tests import vumedra_util as vx
from tests.plain import vumedra_plain as plain


# --------------------------------------------------------------------------- configuration
@pytest.mark.parametrize("make", [vx.config_a, vx.config_b, vx.config_c, vx.config_d])
def test_declared_tensors_are_the_checkpoint_format(make):
    raw = make()
    _, _, spec = resolve(raw)
    model = DecoderModel(spec, torch.bfloat16, "cpu")
    assert {k: tuple(v.shape) for k, v in model.weight_decls().items()} == vx.tensor_shapes(raw)
    assert spec.vocab_size == raw["vocab"] and spec.hidden_size == raw["width"] and model.shape_static
    # what enters norms, routers and recurrences besides the products stays in 32-bit
    kept = {k for k, v in model.weight_decls().items() if v.precision == "float32"}
    assert {"final.norm", "l0.norm1", "l0.norm1b"} <= kept
    assert all(k in kept for k in model.weight_decls() if k.rsplit(".", 1)[-1] in ("lam", "router", "b", "norm", "conv"))


def test_cache_needs_follow_the_mixers_and_the_embedding():
    _, _, spec = resolve(vx.config_a())
    model = DecoderModel(spec, torch.bfloat16, "cpu")
    needs = [c.need for c in model.entry_caches]
    f32 = torch.float32
    assert needs[0] == (FixedState((3, 25, 16), f32), FixedState((3,), f32))  # S with its column of ones, the running maximum
    assert needs[1] == PagedKV(2, 32, None)  # keys of 16 and values of 24 in heads of 32
    assert needs[2] == (FixedState((48,), f32), FixedState((3, 48), torch.bfloat16))  # S, the convolution's last inputs
    assert needs[5] == FixedState((1,), torch.int32) and model.embedding_entry == 5  # the token before, behind the run entries
    _, _, spec_b = resolve(vx.config_b())
    assert DecoderModel(spec_b, torch.bfloat16, "cpu").entry_caches[3].need == FixedState((36,), f32)  # one tap: no inputs kept
    groups, states = group_needs(model.entry_caches)
    assert len(groups) == 1 and len(states) == 2 + 2 + 2 + 2 + 1
    cache = CacheManager(model.entry_caches, 4, 16, 2, device=None)
    rc = cache.new_request()
    cache.reserve([(rc, 33)])
    assert cache.num_free() == (1,)
    cache.release(rc)
    assert cache.is_idle()


def test_a_model_without_attention_has_no_pages():
    _, _, spec = resolve(vx.config_d())
    model = DecoderModel(spec, torch.bfloat16, "cpu")
    cache = CacheManager(model.entry_caches, 4, 16, 2, device=None)
    rc = cache.new_request()
    cache.reserve([(rc, 1000)])
    assert cache.num_groups == 0 and rc.num_tokens == 1000 and cache.pages_for(10 ** 6) == ()


@pytest.mark.parametrize("change, error", [
    (lambda r: r["layers"][0].update(type="mamba2"), NotImplementedError),
    (lambda r: r["layers"][0]["mlp"].update(kind="experts"), NotImplementedError),
    (lambda r: r["layers"][1]["mixer"].update(kv_heads=4), ValueError),
    (lambda r: r["layers"][1]["mixer"]["q_temp"].update(every=0), ValueError),
    (lambda r: r["layers"][0]["mixer"].update(gate_cap=0.0), ValueError),
    (lambda r: r["layers"][2]["mixer"].update(blocks=5), ValueError),
    (lambda r: r["layers"][2]["mixer"].update(conv=0), ValueError),
    (lambda r: r["layers"][1]["mlp"]["router"].update(top=7), ValueError),
    (lambda r: r["embedding"]["bigram"].update(buckets=0), ValueError),
    (lambda r: r.update(layers=[]), ValueError),
    (lambda r: r.pop("norm"), KeyError),
])
def test_refused_configurations(change, error):
    raw = vx.config_a()
    change(raw)
    with pytest.raises(error):
        resolve(raw)


def test_the_preset_and_optional_tensors():
    _, _, spec = resolve(preset("vumedra-tiny"))
    assert [layer.mixer.kind for layer in spec.layers] == ["rglru", "gqa_attention", "mlstm", "rglru"]
    _, _, spec_b = resolve(vx.config_b())
    assert set(spec_b.optional_tensors) == {"l1.norm2", "l1.norm2b"}  # the layer without a feed-forward


# --------------------------------------------------------------------------- the oracle against other statements
def test_bigram_rows_and_sinusoid():
    assert plain.bigram_rows([5, 7, 7, 0], 10, 3, 4).tolist() == [10, (15 + 28) % 10, (21 + 28) % 10, 21 % 10]
    assert plain.bigram_rows([9], 10, 3, 4).tolist() == [10]
    s = plain.sinusoid(torch.arange(50), 6)
    for p in (0, 1, 49):
        for i in range(3):
            ang = p * 10000.0 ** (-2.0 * i / 6)
            assert abs(s[p, 2 * i] - math.sin(ang)) < 1e-5 and abs(s[p, 2 * i + 1] - math.cos(ang)) < 1e-5
    assert plain.sinusoid(torch.arange(3), 5).shape == (3, 5)


def test_sink_softmax_is_a_softmax_with_one_more_key_of_score_zero():
    torch.manual_seed(0)
    s = torch.randn(4, 9) * 5
    s[1] = -40.0  # everything far below the sink
    want = torch.softmax(torch.cat((s, torch.zeros(4, 1)), -1).double(), -1)[:, :-1]
    assert (plain.sink_softmax(s).double() - want).abs().max() < 1e-6
    assert plain.sink_softmax(s)[1].sum() < 1e-15


def test_query_temperature_steps_at_multiples_of_every():
    f = plain.query_temperature(torch.arange(20), 0.5, 4)
    for p in range(20):
        assert abs(f[p] - (1 + 0.5 * math.log(math.floor((p + 1) / 4) + 1))) < 1e-6
    assert f[2] == 1.0 and f[3] > 1.0  # position 3 is the fourth token


def test_matrix_memory_equals_its_quadratic_form():
    """Without the running maximum: weights exp(i_s + sum of f between s and t), numerator and normaliser over all s <= t,
    the denominator max(|n . q|, 1) + 1e-6 exp(m) in unscaled terms."""
    torch.manual_seed(1)
    t, h, dk, dv = 13, 3, 4, 5
    q, k, v = (torch.randn(t, h, d, dtype=torch.float64) for d in (dk, dk, dv))
    i = 3.0 * torch.randn(t, h, dtype=torch.float64)
    f = -torch.rand(t, h, dtype=torch.float64) * 2.0
    got = plain.mlstm_memory(q, k, v, i, f)
    cum = torch.cumsum(f, 0)
    for hd in range(h):
        m = 0.0
        for x in range(t):
            m = max(f[x, hd] + m, i[x, hd])
            w = torch.exp(i[: x + 1, hd] + cum[x, hd] - cum[: x + 1, hd])
            s = (k[: x + 1, hd] @ q[x, hd]) * w
            want = (s @ v[: x + 1, hd]) / (max(abs(s.sum().item()), 1.0) + 1e-6 * math.exp(m))
            assert (got[x, hd] - want).abs().max() < 1e-9


def test_gates_are_capped_and_the_forget_gate_is_a_log_sigmoid():
    i, f = plain.mlstm_gates(torch.tensor([100.0, -100.0, 0.5]), torch.tensor([100.0, -100.0, 0.5]), 4.0)
    assert torch.allclose(i, torch.tensor([4.0, -4.0, 4.0 * math.tanh(0.125)]))
    assert torch.allclose(f, torch.nn.functional.logsigmoid(torch.tensor([4.0, -4.0, 4.0 * math.tanh(0.125)])), atol=1e-6)


def test_gated_linear_recurrence_equals_its_sum():
    torch.manual_seed(2)
    t, c = 12, 5
    u, r, g = torch.randn(t, c), torch.rand(t, c), torch.rand(t, c)
    lam = torch.randn(c)
    got = plain.rglru_scan(u, r, g, lam)
    log_a = -8.0 * r.double() * torch.nn.functional.softplus(lam.double())
    cum = torch.cumsum(log_a, 0)
    for x in range(t):
        w = torch.exp(cum[x][None] - cum[: x + 1]) * torch.sqrt(1 - torch.exp(2 * log_a[: x + 1]))
        assert (got[x].double() - (w * g[: x + 1].double() * u[: x + 1].double()).sum(0)).abs().max() < 1e-5


def test_block_linear_is_a_block_diagonal_matrix():
    torch.manual_seed(3)
    w, b, u = torch.randn(3, 4, 4), torch.randn(3, 4), torch.randn(6, 12)
    full = torch.block_diag(*w)
    assert (plain.block_linear(u, w, b) - (u @ full.T + b.reshape(-1))).abs().max() < 1e-5


def test_an_expert_weighed_at_its_input_is_weighed_by_the_square_at_its_output():
    torch.manual_seed(4)
    w = {"up": torch.randn(7, 5), "down": torch.randn(5, 7)}
    x = torch.randn(3, 5)
    for g in (0.1, 0.5, 1.0):
        assert torch.allclose(plain.expert(g * x, w, "", torch.float32), g * g * plain.expert(x, w, "", torch.float32), atol=1e-5)


def test_router_takes_the_largest_sigmoids_as_they_are():
    w = {"router": torch.tensor([[1.0], [-2.0], [0.5], [3.0]])}
    chosen, weights = plain.route(torch.tensor([[1.0], [-1.0]]), w, "", 2, torch.float32)
    assert chosen.tolist() == [[3, 0], [1, 2]]
    assert np.allclose(weights[0].numpy(), [1 / (1 + math.exp(-3)), 1 / (1 + math.exp(-1))])
