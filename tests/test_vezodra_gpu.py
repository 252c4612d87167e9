"""The Vezodra cases of ``test_vezodra.py`` on the CUDA kernels (``csrc/parallel_mixers.cu``, ``csrc/seq_mixers.cu``): the same
functions, collected here under the ``gpu`` marker; the ops take their kernel branch because their tensors live on the device."""

import pytest
import torch

from test_vezodra import *  # noqa: F401,F403  (collects every test of that module again)
from test_vezodra import (ATT, ODD, PAIR, O, P, _removal_case, _removal_oracle, _removal_run, close, feed, make_cfg, make_engine,
                          row_errors, tokens)
from shuffle_exchange_b200.native import lib as _lib

pytestmark = pytest.mark.gpu


def test_the_kernels_ran():
    before = _lib.launch_count
    x = torch.ones(3, 16, device="cuda")
    P.stream_add(x, P.StreamSum(y=torch.ones(3, 16, device="cuda")), 1e-5, torch.float32)
    assert _lib.launch_count == before + 1
    assert torch.allclose(x, torch.full_like(x, 2.0))


WIDE = make_cfg([
    dict(ATT, mixer={"dim": 64, "heads": 4, "kv_heads": 2, "rot": {"base": 1e4, "dims": 32}, "scale": 0.12, "vdim": 64},
         mlp={"ff": 192, "kind": "dense"}),
    dict(PAIR, mixer={"left": {"dim": 32, "heads": 4, "kv_heads": 1, "mask": {"size": 40},
                               "rot": {"base": 5e3, "dims": 32, "scaling": {"factor": 4.0}}, "scale": 0.18, "vdim": 64},
                      "right": {"dim": 64, "heads": 3}}, mlp={"ff": 128, "kind": "dense"})],
    width=128, vocab=100, taps=4, loop=(1, 2, 2))


def test_prompts_on_the_tiled_and_vector_kernels_in_both_precisions():
    W = O.random_weights(WIDE, seed=31, rank=24)
    toks = tokens(150, WIDE["vocab"], 32)
    want = O.forward(WIDE, W, toks)
    eng = make_engine(WIDE, W, dtype=torch.bfloat16, max_tokens=256, blocks=128)
    for uid, sizes in ((1, [len(toks)]), (2, [70, 1, 33, 1, 1])):
        assert row_errors(feed(eng, uid, toks, sizes), want).max() < 0.06
    eng32 = make_engine(WIDE, W, dtype=torch.float32, max_tokens=256, blocks=128)
    close(feed(eng32, 1, toks, [len(toks)]), want)
    close(feed(eng32, 2, toks, [70, 1, 33, 1, 1]), want)


def test_a_prompt_long_enough_for_the_multi_token_form_of_the_operand_kernel():
    W = O.random_weights(WIDE, seed=33, rank=24)
    toks = tokens(600, WIDE["vocab"], 34)
    want = O.forward(WIDE, W, toks)
    eng = make_engine(WIDE, W, max_tokens=640, blocks=256)
    close(feed(eng, 1, toks, [593, 1, 1, 5]), want)


@pytest.mark.parametrize("H,n,rank,T", [(2, 64, 16, 517), (1, 33, 5, 515), (2, 128, 64, 513), (1, 256, 8, 600)])
def test_delta_rule_over_long_prompts(H, n, rank, T):
    proj, B, P_ = _removal_case(H, n, rank, T, n)
    want = _removal_oracle(proj, B, P_, H, n, rank)
    for cuts in ([T], [T - 3, 1, 1, 1]):
        got = _removal_run(proj, B, P_, H, n, rank, cuts)
        assert torch.allclose(got, want, atol=5e-4, rtol=1e-3), float((got - want).abs().max())


def test_other_sizes_in_bf16():
    """Widths and head sizes that are not multiples of 8 take the scalar forms of the kernels and the library products; 16-bit
    serving must still follow the exact evaluation."""
    for cfg, rank in ODD:
        W = O.random_weights(cfg, seed=8, rank=rank)
        toks = tokens(40, cfg["vocab"], 9)
        want = O.forward(cfg, W, toks)
        eng = make_engine(cfg, W, dtype=torch.bfloat16, block_size=8)
        for uid, sizes in ((1, [len(toks)]), (2, [19, 1, 2])):
            err = row_errors(feed(eng, uid, toks, sizes), want)
            assert err.median() < 0.03 and err.max() < 0.15, err


def test_wide_streams():
    """Rows of more than 8192 channels and rows that are not whole 16-byte words take the element-wise forms."""
    from test_vezodra import test_sums_norms_and_input_filter as case
    for W, taps in ((8200, 4), (4096, 4), (8192, 3), (1001, 2)):
        case(W, taps, True)


def test_queued_batches_never_share_a_staging_buffer():
    """Forwards are queued without a synchronisation: while a long kernel holds the stream back, later batches must not
    overwrite the metadata of the uploads that still wait behind it."""
    from shuffle_exchange_b200.inference.v2.ragged.ragged_wrapper import RaggedBatchWrapper

    class _Seq:
        seen_tokens = 0

        def kv_blocks(self):
            return torch.zeros(1, dtype=torch.int32)
    wrap = RaggedBatchWrapper(16, 2, 4, device="cuda")
    big = torch.randn(4096, 4096, device="cuda")
    for _ in range(20):
        big = big @ big / 64.0
    got = []
    for i in range(3):
        wrap.clear()
        wrap.insert_sequence(_Seq(), torch.full((5,), 100 + i, dtype=torch.int32))
        wrap.finalize()
        got.append(wrap.input_ids().clone())
    torch.cuda.synchronize()
    assert [int(g[0]) for g in got] == [100, 101, 102] and all(bool((g == g[0]).all()) for g in got)
