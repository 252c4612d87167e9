"""The Sudupel cases of ``test_sudupel.py`` on the CUDA kernels (``csrc/gated_mixers.cu``, ``csrc/seq_mixers.cu``,
``csrc/parallel_mixers.cu``, ``csrc/moe_ragged.cu``): the same functions, collected here under the ``gpu`` marker; the ops take
their kernel branch because their tensors live on the device."""

import copy

import pytest
import torch

from test_sudupel import *  # noqa: F401,F403  (collects every test of that module again)
from test_sudupel import (LIGHT, MOE, ODD, UNIT, WIN, Gt, M, O, _unit, _unit_oracle, _unit_step, _walk, close, feed, make_cfg,
                          make_engine, row_errors, tokens)
from shuffle_exchange_b200.native import lib as _lib

pytestmark = pytest.mark.gpu


def test_the_kernels_ran():
    before = _lib.launch_count
    y = Gt.silu_columns(torch.ones(3, 16, device="cuda"))
    assert _lib.launch_count == before + 1
    assert torch.allclose(y, torch.full_like(y, 0.7310586))


def _wide():
    unit, win, light = copy.deepcopy(UNIT), copy.deepcopy(WIN), copy.deepcopy(LIGHT)
    unit["mixer"]["left"].update(dim=64, heads=4, kv_heads=2, vdim=64, scale=0.12)
    unit["mixer"]["left"]["rot"]["dims"] = 32
    unit["mixer"]["right"] = {"width": 192, "blocks": 2, "conv": 4}
    unit["mlp"] = {"kind": "moe", "expert": {"ff": 96}, "router": {"experts": 8, "groups": {"count": 4, "keep": 2}, "top": 2}}
    win["mixer"]["left"].update(dim=32, heads=4, kv_heads=1, vdim=64, scale=0.18, mask={"size": 40})
    win["mixer"]["left"]["rot"]["dims"] = 32
    win["mixer"]["right"] = {"dim": 64, "heads": 3, "vdim": 32, "tau": 16.0}
    win["mlp"] = {"ff": 128, "kind": "dense", "limit": 1.0}
    light["mixer"] = {"dim": 64, "heads": 4, "vdim": 32, "decay": [0.6, 0.9, 0.99, 0.999]}
    return make_cfg([light, win, unit], width=128, vocab=100)


WIDE = _wide()


def test_prompts_on_the_tiled_and_vector_kernels_in_both_precisions():
    W = O.random_weights(WIDE, seed=31, rank=24)
    toks = tokens(150, WIDE["vocab"], 32)
    want = O.forward(WIDE, W, toks)
    eng = make_engine(WIDE, W, dtype=torch.bfloat16, max_tokens=256, blocks=128)
    for uid, sizes in ((1, [len(toks)]), (2, [70, 1, 33, 1, 1])):
        err = row_errors(feed(eng, uid, toks, sizes), want)
        assert err.median() < 0.03 and err.max() < 0.3
    eng32 = make_engine(WIDE, W, dtype=torch.float32, max_tokens=256, blocks=128)
    close(feed(eng32, 1, toks, [len(toks)]), want)
    close(feed(eng32, 2, toks, [70, 1, 33, 1, 1]), want)


def test_a_prompt_long_enough_for_the_multi_row_forms():
    W = O.random_weights(WIDE, seed=33, rank=24)
    toks = tokens(1100, WIDE["vocab"], 34)
    want = O.forward(WIDE, W, toks)
    eng = make_engine(WIDE, W, max_tokens=1152, blocks=600)
    close(feed(eng, 1, toks, [1093, 1, 1, 5]), want)
    close(feed(eng, 2, toks, [3, 600, 497]), want)


@pytest.mark.parametrize("N,blocks,taps,T", [(512, 2, 4, 1030), (192, 4, 3, 517), (70, 1, 2, 600), (96, 32, 4, 300)])
def test_recurrent_unit_over_long_prompts(N, blocks, taps, T):
    g = torch.Generator().manual_seed(N)
    U, x, y = _unit(N, blocks, taps, N), torch.randn(T, N, generator=g), torch.randn(T, N, generator=g)
    want = _unit_oracle(U, x, y)
    for cuts in ([T], [T - 3, 1, 1, 1], [31, 33, 65, T - 129]):
        state, conv = torch.full((3, N), 5.0, device="cuda"), torch.full((3, taps - 1, N), 5.0, device="cuda")
        got = _walk(lambda lo, n, info: _unit_step(U, x[lo: lo + n].cuda(), y[lo: lo + n].cuda(), state, conv, info,
                                                   torch.zeros(n, dtype=torch.int32, device="cuda"), n == 1), T, cuts)
        assert torch.allclose(got, want, atol=5e-5, rtol=1e-3), float((got - want).abs().max())


@pytest.mark.parametrize("Hn,Hv,rank,T", [(128, 256, 16, 520), (33, 7, 5, 515), (256, 256, 64, 600)])
def test_operands_over_long_prompts(Hn, Hv, rank, T):
    g = torch.Generator().manual_seed(Hn)
    x = torch.randn(T, 2 * Hn + Hv + rank, generator=g)
    w2, b = torch.randn(rank, Hn, generator=g), torch.randn(Hn, generator=g)
    a = (0, Hn, 2 * Hn, 2 * Hn + Hv)
    want = Gt.decay_prepare(x, *a, w2, b, Hn, Hv, 0.3, 7.0)
    got = Gt.decay_prepare(x.cuda(), *a, w2.cuda(), b.cuda(), Hn, Hv, 0.3, 7.0)
    for u, v in zip(got, want):
        assert torch.allclose(u.cpu(), v, atol=1e-5)


def test_other_sizes_in_bf16():
    """Widths and head sizes that are not multiples of 8 take the scalar forms of the kernels and the library products; 16-bit
    serving must still follow the exact evaluation (a close choice of experts may fall the other way in a few rows)."""
    for cfg, rank in ODD:
        W = O.random_weights(cfg, seed=8, rank=rank)
        toks = tokens(40, cfg["vocab"], 9)
        want = O.forward(cfg, W, toks)
        eng = make_engine(cfg, W, dtype=torch.bfloat16, block_size=8)
        for uid, sizes in ((1, [len(toks)]), (2, [19, 1, 2])):
            err = row_errors(feed(eng, uid, toks, sizes), want)
            assert err.median() < 0.05 and (err > 0.3).sum() <= 4, err


def test_wide_streams():
    """Rows of more than 8192 channels and rows that are not whole 16-byte words take the element-wise forms."""
    from test_sudupel import test_gated_norm_into_a_slice_of_wider_rows as gate_case
    from test_sudupel import test_norms_before_and_after_a_sublayer_with_weights_around_zero as case
    for W in (8200, 4096, 8192, 1001):
        case(W)
        gate_case(W, W, W, True, False)
