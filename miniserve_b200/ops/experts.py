"""Python faces of the kernels in ``csrc/routed_experts.cu``: a router's choice, the plan that sorts a step's
(token, choice) pairs by expert, the experts' products over the sorted rows, and the weighted sum."""

from __future__ import annotations

import os

import torch

from . import native
from .mixers import _dt, _f32, _ptr, _rows, _stream

ACTIVATIONS = {"silu": 0, "gelu_tanh": 1, "relu_squared": 2, "clamped_glu": 3}
NO_CLAMPS = (-1.0, 1.0, 0.0)  # (limit, alpha, shift) of a clamped GLU; other activations do not read them
SCORES = {"softmax": 0, "sigmoid": 1}
TILE_ROWS = 64       # sorted rows per tile of the float32 and mma.sync products
TC_TILE_ROWS = 128   # of the products on the tcgen05 tensor cores
TC_FEW_ROWS = 32     # of the same where an expert has a few rows (decode steps)
TC_EXPERTS = os.environ.get("MINISERVE_TC_EXPERTS", "1") != "0"  # bfloat16 experts on the tcgen05 kernel where it takes the shape


def tc_experts_ok(dtype, hidden: int, inter: int, activation: str) -> bool:
    """Whether the experts' products of this shape run on the tcgen05 kernel (``csrc/gemm_tc.cu``, the grouped form):
    bfloat16, an activation that the kernel has as an epilogue (SiLU times the up half, the clamped GLU, or the square of relu without a
    gate), rows that are multiples of 16 bytes."""
    return TC_EXPERTS and dtype == torch.bfloat16 and activation in ("silu", "relu_squared", "clamped_glu") and hidden % 8 == 0 and inter % 8 == 0


def tc_tile_rows(slots: int, experts: int) -> int:
    """Rows per tile of the tcgen05 products for a step of ``slots`` (token, choice) pairs."""
    return TC_FEW_ROWS if slots <= FEW_ROWS_PER_EXPERT * experts else TC_TILE_ROWS


FEW_ROWS_PER_EXPERT = 16  # up to so many rows per expert on average: tiles of TC_FEW_ROWS


def expert_route(idx, wgt, x, router, correction, top: int, group_count: int, group_keep: int, weight_scale: float,
                 renormalize: bool, stream=None, logit_bias=None, gate_w=None, gate_out=None, score: str = "softmax",
                 square_weights: bool = False, group_best: int = 1, renorm_eps: float = 0.0) -> None:
    """idx [T, top] int32 and wgt [T, top] float32: each token's chosen router outputs and their weights.
    Logits ``x router^T`` in float32 (``router`` [R, K] float32), scores their softmax, choice scores the scores plus
    ``correction`` [R] (float32, or None); the R outputs form ``group_count`` equal groups of neighbours of which the
    ``group_keep`` with the largest sum of their ``group_best`` largest choice scores can be chosen from; weights are the chosen scores (without
    the correction) times ``weight_scale``, divided by their sum (+ ``renorm_eps``) if ``renormalize`` (which makes them the softmax over
    the chosen logits alone). Ties go to the lower index. ``logit_bias`` [R] float32 is added to the logits themselves.
    ``gate_w`` [K] float32 with ``gate_out`` [T] float32: gate_out[t] = sigmoid(x[t] . gate_w), from the same staged input.
    ``score`` = ``sigmoid``: the scores are the logits' sigmoids. ``square_weights``: the final weights are squared."""
    t, k = x.shape
    r = router.shape[0]
    _f32(router, correction, wgt, logit_bias, gate_w, gate_out)
    assert (gate_w is None) == (gate_out is None) and (gate_w is None or (gate_w.numel() == k and gate_out.numel() >= t))
    assert logit_bias is None or logit_bias.numel() == r
    assert router.shape == (r, k) and idx.shape == (t, top) and wgt.shape == (t, top) and idx.dtype == torch.int32
    assert idx.is_contiguous() and (correction is None or correction.numel() == r)
    native.experts_check(native.experts().ms_expert_route(
        _ptr(idx), _ptr(wgt), _ptr(x), _rows(x), _ptr(router), _ptr(correction), t, k, r, top, group_count, group_keep,
        float(weight_scale), int(renormalize), _dt(x.dtype), _stream(stream), _ptr(logit_bias), _ptr(gate_w), _ptr(gate_out),
        SCORES[score], int(square_weights), int(group_best), float(renorm_eps)))


def expert_max_tiles(slots: int, experts: int, tile_rows: int = TILE_ROWS) -> int:
    """The most tiles of ``tile_rows`` sorted rows a step of ``slots`` (token, choice) pairs over ``experts`` experts can have."""
    return int(native.experts().ms_expert_max_tiles_of(slots, experts, tile_rows))


def expert_plan(pos, perm, offsets, tiles, meta, idx, experts: int, stream=None, tile_rows: int = TILE_ROWS) -> None:
    """Sorts the slots of ``idx`` [T, top] by expert, on the device: ``pos`` [T * top] the sorted row of a slot (-1: the
    slot's choice is not one of the ``experts`` experts with tensors), ``perm`` [T * top] the slot of a sorted row,
    ``offsets`` [experts + 1], ``tiles`` [max_tiles, 2] = (expert, first row), ``meta`` [2] = (tiles, sorted rows)."""
    slots = idx.numel()
    for a in (pos, perm, offsets, tiles, meta, idx):
        assert a.dtype == torch.int32 and a.is_contiguous() and a.is_cuda
    assert pos.numel() == slots and perm.numel() == slots and offsets.numel() == experts + 1 and meta.numel() >= 2
    assert tiles.numel() >= 2 * expert_max_tiles(slots, experts, tile_rows)
    native.experts_check(native.experts().ms_expert_plan_of(_ptr(pos), _ptr(perm), _ptr(offsets), _ptr(tiles), _ptr(meta), _ptr(idx),
                                                            slots, experts, tile_rows, _stream(stream)))


def expert_gather(xs, x, perm, meta, top: int, stream=None) -> None:
    """xs [T * top, K] bfloat16, row r = x[perm[r] // top] for the plan's sorted rows (the rows behind them stay as they are)."""
    slots, k = xs.shape
    assert x.shape[1] == k and xs.is_contiguous() and xs.dtype == x.dtype == torch.bfloat16
    native.experts_check(native.experts().ms_expert_gather(_ptr(xs), _ptr(x), _rows(x), _ptr(perm), _ptr(meta), top, slots, k,
                                                           _stream(stream)))


def expert_products_tc(out, a, w, tiles, meta, offsets, gated: bool, stream=None, relu_squared: bool = False, clamps=None,
                       tile_rows: int = TC_TILE_ROWS) -> None:
    """The experts' products over sorted rows on the tcgen05 tensor cores (the plan's tiles have ``tile_rows`` rows: ``tc_tile_rows``).
    ``gated``: out [S, I] bfloat16 = silu(a W_gate[e]^T) * (a W_up[e]^T) (or with ``clamps`` = (limit, alpha, shift) the clamped GLU of the two) with ``w`` [E, 2 I, K]; else out [S, N] float32 =
    a W[e]^T with ``w`` [E, N, K] (``relu_squared``: bfloat16, the square of its relu). ``a`` [S, K] bfloat16 in sorted order."""
    from . import device_status

    slots, n = out.shape
    e, w_rows, k = w.shape
    assert a.shape == (slots, k) and a.is_contiguous() and w.is_contiguous() and out.is_contiguous()
    assert a.dtype == w.dtype == torch.bfloat16 and w_rows == (2 * n if gated else n)
    assert out.dtype == (torch.bfloat16 if gated or relu_squared else torch.float32) and not (gated and relu_squared)
    lib = native.gemm_tc()
    mode = 2 if relu_squared else (3 if clamps is not None else 1) if gated else 0
    native.kernel_check(lib.ms_gemm_tc_experts_bf16(_ptr(out), _ptr(a), _ptr(w), slots, n, k, e, mode, _ptr(tiles), _ptr(meta),
                                                    _ptr(offsets), tile_rows, expert_max_tiles(slots, e, tile_rows), *map(float, clamps or NO_CLAMPS),
                                                    _ptr(device_status(a.device)), _stream(stream)),
                        lib=lib, errfn="ms_gemm_tc_last_error")


def expert_gate_up(out, x, w_gate_up, perm, top: int, tiles, meta, offsets, activation: str, stream=None, clamps=None) -> None:
    """out [T * top, I] (the run's dtype), row r = act(W_gate[e] h) * (W_up[e] h) (``clamped_glu``: the clamped GLU of the two with
    ``clamps`` = (limit, alpha, shift)) with h = x[perm[r] // top] and e the
    expert whose sorted rows hold r; ``w_gate_up`` [E, 2 I, K]: an expert's gate rows, then its up rows."""
    slots, inter = out.shape
    e, two_i, k = w_gate_up.shape
    assert two_i == 2 * inter and x.shape[1] == k and out.is_contiguous() and w_gate_up.is_contiguous()
    assert out.dtype == x.dtype == w_gate_up.dtype
    native.experts_check(native.experts().ms_expert_gemm(
        _ptr(out), _ptr(x), _rows(x), _ptr(perm), top, _ptr(w_gate_up), _ptr(tiles), _ptr(meta), _ptr(offsets),
        expert_max_tiles(slots, e), inter, k, 1, ACTIVATIONS[activation], *map(float, clamps or NO_CLAMPS), _dt(x.dtype), _stream(stream)))


def expert_up(out, x, w_up, perm, top: int, tiles, meta, offsets, activation: str, stream=None) -> None:
    """out [T * top, I] (the run's dtype), row r = act(W_up[e] h) with h = x[perm[r] // top]; ``w_up`` [E, I, K] (experts without a gate)."""
    slots, inter = out.shape
    e, i, k = w_up.shape
    assert i == inter and x.shape[1] == k and out.is_contiguous() and w_up.is_contiguous() and out.dtype == x.dtype == w_up.dtype
    native.experts_check(native.experts().ms_expert_gemm(
        _ptr(out), _ptr(x), _rows(x), _ptr(perm), top, _ptr(w_up), _ptr(tiles), _ptr(meta), _ptr(offsets),
        expert_max_tiles(slots, e), inter, k, 2, ACTIVATIONS[activation], *NO_CLAMPS, _dt(x.dtype), _stream(stream)))


def expert_down(out, act, w_down, tiles, meta, offsets, stream=None) -> None:
    """out [T * top, H] float32, row r = W_down[e] act[r] over the sorted rows; ``w_down`` [E, H, I]."""
    slots, hidden = out.shape
    e, h, inter = w_down.shape
    _f32(out)
    assert h == hidden and act.shape == (slots, inter) and act.is_contiguous() and w_down.is_contiguous() and act.dtype == w_down.dtype
    native.experts_check(native.experts().ms_expert_gemm(
        _ptr(out), _ptr(act), inter, None, 1, _ptr(w_down), _ptr(tiles), _ptr(meta), _ptr(offsets),
        expert_max_tiles(slots, e), hidden, inter, 0, 0, *NO_CLAMPS, _dt(act.dtype), _stream(stream)))


def expert_combine(out, y, x, idx, wgt, pos, experts: int, stream=None, shared=None, shared_gate=None) -> None:
    """out[t] = sum over the token's choices, in their order, of wgt * (y[pos] for an expert with tensors, x[t] for a
    router output from ``experts`` on: an identity expert); float32 sum, one rounding. ``shared`` [T, H] (the run's
    dtype): the output of an expert that every token uses, added times ``shared_gate`` [T] float32 (or once)."""
    t, hidden = out.shape
    top = idx.shape[1]
    _f32(y, wgt)
    assert out.is_contiguous() and x.shape == (t, hidden) and x.dtype == out.dtype and y.shape[1] == hidden
    assert shared is None or (shared.shape == (t, hidden) and shared.dtype == out.dtype and shared.is_contiguous())
    _f32(shared_gate)
    native.experts_check(native.experts().ms_expert_combine(
        _ptr(out), _ptr(y), _ptr(x), _rows(x), _ptr(idx), _ptr(wgt), _ptr(pos), t, hidden, top, experts, _dt(out.dtype),
        _stream(stream), _ptr(shared), _ptr(shared_gate)))
