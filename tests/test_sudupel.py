"""Sudupel in the ragged engine against the plain evaluation in ``sudupel_oracle.py`` (float64, whole sequences, no cache):
every mechanism alone, prefill against token-by-token decoding, prompt portions down to two tokens, unequal batches, reuse of
cache pages and state slots, window edges, the softmax's added one, keys and writes far back, the first tokens, long decoding,
expert choices, other sizes, and greedy generation through the scheduler.  Runs on the PyTorch branch of every op without a GPU;
``test_sudupel_gpu.py`` runs the same cases on the CUDA kernels."""
import copy
import json
import math
import os
import struct
import subprocess
import sys

import pytest
import torch

import sudupel_oracle as O
from shuffle_exchange_b200.inference.v2.config_v2 import RaggedInferenceEngineConfig
from shuffle_exchange_b200.inference.v2.engine_factory import build_engine_from_state_dict
from shuffle_exchange_b200.inference.v2.inference_utils import ActivationType, DtypeEnum
from shuffle_exchange_b200.inference.v2.kernels import gated_ops as Gt
from shuffle_exchange_b200.inference.v2.kernels import mixer_ops as M
from shuffle_exchange_b200.inference.v2.kernels import parallel_ops as P
from shuffle_exchange_b200.inference.v2.modules import heuristics
from shuffle_exchange_b200.inference.v2.modules.configs import (DSMoEConfig, DSSelfAttentionConfig, MaskingType,
                                                               PositionalEmbeddingType, RotaryScalingConfig, RotateHalfConfig)
from shuffle_exchange_b200.inference.v2.modules.implementations import scaled_rotary_table
from shuffle_exchange_b200.inference.v2.ragged.ragged_manager import DSStateManagerConfig
from shuffle_exchange_b200.inference.v2.scheduler import generate
from shuffle_exchange_b200.ops import moe_ops

DEV = "cuda" if torch.cuda.is_available() else "cpu"
F64 = torch.float64

DENSE = {"ff": 24, "kind": "dense", "limit": 0.8}
MOE = {"kind": "moe", "expert": {"ff": 12}, "router": {"experts": 12, "groups": {"count": 4, "keep": 2}, "top": 3}}
LIGHT = {"type": "lightning", "mixer": {"dim": 8, "heads": 3, "vdim": 12, "decay": [0.55, 0.9, 0.995]}, "mlp": DENSE}
UNIT = {"type": "parallel",
        "mixer": {"left": {"dim": 8, "heads": 4, "kv_heads": 2, "vdim": 6, "scale": 0.4,
                           "rot": {"base": 300.0, "dims": 6, "scaling": {"factor": 3.0, "original": 64, "fast": 8.0, "slow": 1.0}}},
                  "right": {"width": 20, "blocks": 5, "conv": 3}, "left_scale": 0.7, "right_scale": 0.9}, "mlp": MOE}
WIN = {"type": "parallel_2",
       "mixer": {"left": {"dim": 8, "heads": 6, "kv_heads": 3, "vdim": 10, "conv": 4, "mask": {"size": 7}, "scale": 0.5,
                          "rot": {"base": 90.0, "dims": 8}},
                 "right": {"dim": 4, "heads": 3, "vdim": 8, "tau": 5.0}, "left_scale": 1.3, "right_scale": 0.4}, "mlp": MOE}


def make_cfg(layers, width=24, vocab=53, eps=1e-5, scale=3.0, cap=6.0):
    return {"architecture": "Sudupel", "embedding": {"scale": scale}, "layers": copy.deepcopy(layers), "logit_softcap": cap,
            "norm": {"eps": eps}, "vocab": vocab, "width": width}


STACK = make_cfg([LIGHT, WIN, dict(UNIT, mlp=None), dict(WIN, mlp=DENSE), UNIT])


def make_engine(cfg, W, dtype=torch.float32, blocks=64, block_size=4, max_live=4, max_tokens=256):
    sm = DSStateManagerConfig(max_tracked_sequences=max_live, max_ragged_sequence_count=max_live,
                              max_ragged_batch_size=max_tokens, max_context=blocks * block_size, num_kv_blocks=blocks)
    return build_engine_from_state_dict(cfg, W, RaggedInferenceEngineConfig(state_manager=sm, kv_block_size=block_size),
                                        dtype=dtype)


def tokens(n, vocab, seed):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def feed(engine, uid, toks, sizes):
    """Give ``toks`` to the engine in portions of the given sizes (cycled); returns the logits of every token."""
    out, lo, i = [], 0, 0
    while lo < len(toks):
        n = min(sizes[i % len(sizes)], len(toks) - lo)
        i += 1
        out.append(engine.put([uid], [torch.tensor(toks[lo: lo + n])], logit_positions=[list(range(n))]))
        lo += n
    return torch.cat(out).double().cpu()


def row_errors(got, want):
    """Difference with the mean over the vocabulary taken off, relative to the spread of the expected logits."""
    d = got - want
    d = d - d.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / want.std()


def close(got, want, tol=2e-4):
    err = row_errors(got, want)
    assert err.max() < tol, f"worst row {int(err.argmax())}: {float(err.max()):.3e}"


CUTS = {"whole": lambda T: [T], "ones": lambda T: [1] * T, "mixed": lambda T: [2, 1, 3, T - 6], "pairs": lambda T: [2] * (T // 2) + [1] * (T % 2)}


@pytest.fixture(scope="module")
def stack():
    W = O.random_weights(STACK, seed=4)
    toks = tokens(47, STACK["vocab"], 5)
    return W, toks, O.forward(STACK, W, toks)


# ------------------------------------------------------------------------------------------------ norms
@pytest.mark.parametrize("W", [40, 24, 7, 1032, 64])
def test_norms_before_and_after_a_sublayer_with_weights_around_zero(W):
    g = torch.Generator().manual_seed(W)
    x, y = torch.randn(9, W, generator=g), torch.randn(9, W, generator=g)
    wa, wb = 0.4 * torch.randn(W, generator=g), 0.4 * torch.randn(W, generator=g)
    r = x.clone().to(DEV)
    out = M.resid_norm_step(r, y.to(DEV), wb.to(DEV), None, wa.to(DEV), 1e-3, torch.float32, w_add=1.0, post_add=1.0)
    want = x.double() + O.rms_norm(y.double(), 1.0 + wb.double(), 1e-3)
    assert torch.allclose(r.double().cpu(), want, atol=1e-5)
    assert torch.allclose(out.double().cpu(), O.rms_norm(want, 1.0 + wa.double(), 1e-3), atol=1e-5)
    r = x.clone().to(DEV)                                          # the other parts of the same kernel
    extra, ls = torch.randn(9, W, generator=g), torch.randn(W, generator=g)
    out = M.resid_norm_step(r, y.to(DEV), None, extra.to(DEV), None, 1e-3, torch.float32, 0.5, True, ls.to(DEV))
    want = (x + 0.5 * y * ls + extra).double()
    assert torch.allclose(r.double().cpu(), want, atol=1e-5) and torch.allclose(out.double().cpu(), want, atol=1e-5)


@pytest.mark.parametrize("C,gs,wlen", [(48, 48, 48), (48, 8, 8), (96, 24, 96), (2048, 2048, 2048), (80, 16, 80), (30, 10, 10), (512, 256, 256),
                                       (512, 64, 64), (64, 32, 32)])
@pytest.mark.parametrize("sigmoid,first", [(True, False), (False, False), (False, True)])
def test_gated_norm_into_a_slice_of_wider_rows(C, gs, wlen, sigmoid, first):
    g = torch.Generator().manual_seed(C + gs)
    T = 5
    y, gate, w = torch.randn(T, C, generator=g), torch.randn(T, C + 8, generator=g), torch.randn(wlen, generator=g)
    wide = torch.full((T, C + 24), 7.0, device=DEV)
    M.group_norm_gate(y.to(DEV), gate.to(DEV)[:, 8:], w.to(DEV), gs, 1e-4, first, torch.float32, sigmoid=sigmoid, out=wide[:, 16: 16 + C],
                      out_scale=0.6)
    Y, G = y.double(), gate[:, 8:].double()
    G = torch.sigmoid(G) if sigmoid else O.silu(G)
    z = (Y * G if first else Y).view(T, -1, gs)
    z = O.rms_norm(z, torch.ones(gs, dtype=F64), 1e-4).view(T, C) * w.double().repeat(C // wlen)
    want = 0.6 * (z if first else z * G)
    assert torch.allclose(wide[:, 16: 16 + C].double().cpu(), want, atol=1e-5)
    assert torch.all(wide[:, :16] == 7.0) and torch.all(wide[:, 16 + C:] == 7.0)


# ------------------------------------------------------------------------------------------------ rotation, attention
@pytest.mark.parametrize("dims,base,scaling", [
    (8, 700.0, None), (64, 1e4, (4.0, 2048, 32.0, 1.0)), (6, 300.0, (3.0, 64, 8.0, 1.0)), (12, 50.0, (1.0, 100, 4.0, 2.0)),
    (2, 10.0, (2.0, 40, 1.0, 1.0)), (16, 1e6, (40.0, 4096, 32.0, 1.0)), (8, 4.0, (2.5, 9, 30.0, 20.0)), (32, 100.0, (2.0, 10 ** 6, 2.0, 1.0))])
def test_frequencies_slowed_by_wavelength(dims, base, scaling):
    rot = {"dims": dims, "base": base}
    sc = None
    if scaling:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
        sc = RotaryScalingConfig(factor=scaling[0], original=scaling[1], fast=scaling[2], slow=scaling[3])
    f, amp = scaled_rotary_table(dims, base, sc)
    assert f.dtype == torch.float32
    assert torch.allclose(f.double(), torch.tensor(O.rotary_frequencies(rot), dtype=F64), rtol=1e-7, atol=0)
    assert amp == pytest.approx(O.rotary_amplitude(rot), rel=1e-12)


def _paged(T, G, d, dv, block_size=4):
    pages = (T + block_size - 1) // block_size
    kc = torch.full((pages + 1, block_size, G, d), 9.0, device=DEV)
    vc = torch.full((pages + 1, block_size, G, dv), 9.0, device=DEV)
    return kc, vc, torch.arange(pages, 0, -1, dtype=torch.int32, device=DEV).view(1, pages)


@pytest.mark.parametrize("Hq,G,d,dv,dims,interleaved,taps", [
    (6, 2, 8, 8, 4, False, 4), (4, 2, 8, 12, 8, False, 3), (3, 1, 5, 3, 4, False, 2), (2, 2, 10, 10, 10, True, 3), (4, 4, 64, 64, 64, False, 4),
    (5, 5, 40, 24, 18, False, 6), (1, 1, 12, 12, 0, False, 1), (2, 1, 130, 7, 126, False, 2), (2, 1, 33, 40, 22, True, 1)])
def test_filter_head_norm_rotation_and_cache_append(Hq, G, d, dv, dims, interleaved, taps):
    g = torch.Generator().manual_seed(d + taps)
    T, C = 19, (Hq + G) * d + G * dv
    x = torch.randn(T, C + 3, generator=g)
    cw = torch.randn(C, taps, generator=g)
    qw, kw = torch.randn(d, generator=g), torch.randn(d, generator=g)
    rot = {"dims": dims, "base": 300.0, "scaling": {"factor": 1.5, "original": 50, "fast": 4.0, "slow": 1.0}}
    freqs, amp = scaled_rotary_table(dims, 300.0, RotaryScalingConfig(factor=1.5, original=50, fast=4.0, slow=1.0))
    f = O.causal_filter(x[:, :C].double(), cw.double())
    q = O.rms_norm(f[:, : Hq * d].reshape(T, Hq, d), qw.double(), 1e-3)
    k = O.rms_norm(f[:, Hq * d: (Hq + G) * d].reshape(T, G, d), kw.double(), 1e-3)
    v = f[:, (Hq + G) * d:].reshape(T, G, dv)
    if interleaved and dims:                                       # the oracle turns halves: reorder its pairs
        order = torch.cat([torch.arange(0, dims, 2), torch.arange(1, dims, 2), torch.arange(dims, d)])
        back = torch.argsort(order)
        q, k = O.rotate(q[..., order], rot)[..., back], O.rotate(k[..., order], rot)[..., back]
    elif dims:
        q, k = O.rotate(q, rot), O.rotate(k, rot)
    for cuts in ([T], [1, 2, 5, 11], [1] * T):
        kc, vc, tables = _paged(T, G, d, dv)
        state = torch.full((3, taps - 1, C), 5.0, device=DEV) if taps > 1 else None
        got, lo = [], 0
        for n in cuts:
            info = torch.tensor([[0, n, lo, 1]], dtype=torch.int32, device=DEV)
            t2s = torch.zeros(n, dtype=torch.int32, device=DEV)
            pos = torch.arange(lo, lo + n, dtype=torch.int32, device=DEV)
            rows = x[lo: lo + n].to(DEV)
            got.append(M.qkv_filter_norm_append(rows, cw.to(DEV), state, info, qw.to(DEV), kw.to(DEV), kc, vc, t2s, pos, tables, Hq, G, d,
                                                dv, 1e-3, True, inv_freq=freqs.to(DEV), interleaved=interleaved, amp=amp).cpu())
            if taps > 1:
                M.conv_state_update(rows[:, :C], state, info)
            lo += n
        assert torch.allclose(torch.cat(got).double(), q, atol=3e-5)
        order = tables[0].long().cpu()
        assert torch.allclose(kc.cpu()[order].reshape(-1, G, d)[:T].double(), k, atol=3e-5)
        assert torch.allclose(vc.cpu()[order].reshape(-1, G, dv)[:T].double(), v, atol=3e-5)
        assert torch.all(kc[0] == 9.0)


@pytest.mark.parametrize("Hq,G,d,dv,dims", [(4, 2, 8, 12, 8), (3, 1, 5, 3, 4), (4, 4, 64, 64, 64), (2, 1, 12, 8, 6)])
def test_whole_row_norm_and_scaled_rotation(Hq, G, d, dv, dims):
    g = torch.Generator().manual_seed(d)
    T, n = 19, Hq * d
    x = torch.randn(T, n + G * (d + dv), generator=g)
    qw, kw = torch.randn(n, generator=g), torch.randn(G * d, generator=g)
    rot = {"dims": dims, "base": 300.0, "scaling": {"factor": 2.5, "original": 50, "fast": 4.0, "slow": 1.0}}
    freqs, amp = scaled_rotary_table(dims, 300.0, RotaryScalingConfig(factor=2.5, original=50, fast=4.0, slow=1.0))
    X = x.double()
    q = O.rotate(O.rms_norm(X[:, :n], qw.double(), 1e-3).view(T, Hq, d), rot)
    k = O.rotate(O.rms_norm(X[:, n: n + G * d], kw.double(), 1e-3).view(T, G, d), rot)
    for cuts in ([T], [1, 2, 5, 11]):
        kc, vc, tables = _paged(T, G, d, dv)
        got, lo = [], 0
        for c in cuts:
            t2s, pos = torch.zeros(c, dtype=torch.int32, device=DEV), torch.arange(lo, lo + c, dtype=torch.int32, device=DEV)
            got.append(P.rope_append(x[lo: lo + c].to(DEV), 0, n, n + G * d, qw.to(DEV), kw.to(DEV), freqs.to(DEV), False, None, kc, vc,
                                     t2s, pos, tables, Hq, G, d, dv, 1e-3, amp).cpu())
            lo += c
        assert torch.allclose(torch.cat(got).double(), q, atol=3e-5)
        assert torch.allclose(kc.cpu()[tables[0].long().cpu()].reshape(-1, G, d)[:T].double(), k, atol=3e-5)


class _Batch:
    """The metadata of one sequence's portion without an engine."""

    def __init__(self, lo, n, tables):
        self._t2s = torch.zeros(n, dtype=torch.int32, device=DEV)
        self._pos = torch.arange(lo, lo + n, dtype=torch.int32, device=DEV)
        self._info = torch.tensor([[0, n, lo, 0]], dtype=torch.int32, device=DEV)
        self._tables = tables

    def token_to_seq(self): return self._t2s
    def token_positions(self): return self._pos
    def block_tables(self): return self._tables
    def seq_info(self): return self._info


def _attention_module(window=0, unit=False, taps=1, H=1, G=1, d=4, dv=None, scale=1.0):
    kw = dict(qkv_conv_taps=taps) if taps > 1 else dict(split_cache=True, unit_sink=unit)
    return heuristics.instantiate_attention(DSSelfAttentionConfig(
        max_tokens=64, n_heads_q=H, n_heads_kv=G, head_size=d, v_head_size=dv or d, max_sequences=4, scale_factor=scale,
        input_dtype=DtypeEnum.fp32, output_dtype=DtypeEnum.fp32,
        masking_type=MaskingType.sliding_window if window else MaskingType.causal,
        masking_args={"size": window} if window else {}, positional_embedding_type=PositionalEmbeddingType.none,
        positional_embedding_config=RotateHalfConfig(rotate_dim=0), **kw), None)


def _run_module(mod, x, cuts, out_scale=1.0):
    c = mod._config
    kc, vc, tables = _paged(x.shape[0], c.n_heads_kv, c.head_size, c.v_head_size)
    n_out = c.n_heads_q * c.v_head_size
    out, lo = [], 0
    for n in cuts:
        wide = torch.full((n, n_out + 5), 7.0, device=DEV)
        mod(x[lo: lo + n].to(DEV).contiguous(), (kc, vc), _Batch(lo, n, tables), None, None, out=wide[:, 3: 3 + n_out], out_scale=out_scale)
        assert torch.all(wide[:, :3] == 7.0) and torch.all(wide[:, 3 + n_out:] == 7.0)
        out.append(wide[:, 3: 3 + n_out].cpu())
        lo += n
    return torch.cat(out).double()


def test_one_joins_the_softmax_denominator_before_any_shift():
    """Scores of -3 with two keys: weights e^-3 / (1 + 2 e^-3); scores of +50: the one does not matter; -200: all vanish.  The result
    is scaled and lands in a column slice."""
    d = 2
    for score in (-3.0, 0.0, 50.0, -200.0):
        x = torch.zeros(2, 3 * d)
        x[:, 0], x[:, d], x[:, 2 * d] = score, 1.0, 3.0
        mod = _attention_module(unit=True, d=d)
        for cuts in ([2], [1, 1]):
            out = _run_module(mod, x, cuts, 0.5)
            e = math.exp(score)
            want = torch.tensor([[1.5 * e / (1 + e), 0.0], [1.5 * 2 * e / (1 + 2 * e), 0.0]], dtype=F64)
            assert torch.allclose(out, want, atol=1e-6), score


# ------------------------------------------------------------------------------------------------ matrix states
def _walk(run, T, cuts, slots=3, slot=1):
    """``run(lo, n, info)`` over the portions of one sequence on a state slot that holds another sequence's numbers."""
    outs, lo = [], 0
    for n in cuts:
        outs.append(run(lo, n, torch.tensor([[0, n, lo, slot]], dtype=torch.int32, device=DEV)).cpu())
        lo += n
    assert lo == T
    return torch.cat(outs).double()


@pytest.mark.parametrize("H,n,dv", [(3, 8, 6), (1, 5, 7), (2, 40, 24), (1, 130, 20), (2, 64, 64), (2, 33, 1), (4, 16, 48)])
@pytest.mark.parametrize("per_channel", [False, True], ids=["fixed_decay", "decay_per_channel"])
def test_decayed_sums_of_outer_products(H, n, dv, per_channel):
    g = torch.Generator().manual_seed(n + dv)
    T = 27
    q, k, v = torch.randn(T, H * n, generator=g), torch.randn(T, H * n, generator=g) / math.sqrt(n), torch.randn(T, H * dv, generator=g)
    decay = torch.rand(T, H * n, generator=g) if per_channel else torch.rand(H, generator=g)
    a = decay.double().view(T, H, n) if per_channel else decay.double().view(1, H, 1).expand(T, H, n)
    want = torch.stack([O.decayed_outer_products(q.double().view(T, H, n)[:, i], k.double().view(T, H, n)[:, i],
                                                 v.double().view(T, H, dv)[:, i], a[:, i]) for i in range(H)], dim=1).reshape(T, H * dv)
    for cuts in ([T], [1] * T, [1, 2, 8, 9, 7], [16, 11]):
        S = torch.full((3, H, dv, n), 5.0, device=DEV)
        got = _walk(lambda lo, c, info: M.linear_recurrence(
            k[lo: lo + c].to(DEV), q[lo: lo + c].to(DEV), v[lo: lo + c].to(DEV),
            (decay[lo: lo + c] if per_channel else decay).contiguous().to(DEV), None, None, S, info, H, H, n, dv, False), T, cuts)
        assert torch.allclose(got, want, atol=1e-4, rtol=1e-4)
        assert torch.all(S[[0, 2]] == 5.0)


def test_what_a_slow_head_wrote_is_read_hundreds_of_tokens_later():
    """Only the first token writes; a head of decay 0.999 still reads it at token 400 and one of 0.5 reads nothing."""
    T, n = 400, 4
    k, q, v = torch.zeros(T, 2 * n), torch.zeros(T, 2 * n), torch.zeros(T, 2 * n)
    k[0, 0] = k[0, n] = 1.0
    v[0] = torch.arange(1.0, 9.0)
    q[T - 1, 0] = q[T - 1, n] = 1.0
    decay = torch.tensor([0.999, 0.5])
    for cuts in ([T], [200, 2] + [1] * 198):
        S = torch.zeros(2, 2, n, n, device=DEV)
        got = _walk(lambda lo, c, info: M.linear_recurrence(k[lo: lo + c].to(DEV), q[lo: lo + c].to(DEV), v[lo: lo + c].to(DEV),
                                                            decay.to(DEV), None, None, S, info, 2, 2, n, n, False), T, cuts)
        assert torch.allclose(got[T - 1, :n], 0.999 ** 399 * torch.arange(1.0, 5.0, dtype=F64), rtol=1e-4)
        assert got[T - 1, n:].abs().max() < 1e-20


@pytest.mark.parametrize("H,n,dv,rank,T", [(3, 8, 6, 6, 11), (1, 5, 7, 1, 9), (2, 16, 40, 16, 5), (2, 33, 3, 20, 3)])
def test_operands_and_decay_per_key_channel(H, n, dv, rank, T):
    g = torch.Generator().manual_seed(n)
    Hn, Hv = H * n, H * dv
    cols = [8 * ((w + 7) // 8) for w in (Hn, Hn, Hv)]
    q0, k0, v0, low0 = 0, cols[0], cols[0] + cols[1], sum(cols)
    x = torch.randn(T, low0 + rank, generator=g)
    w2, b = torch.randn(rank, Hn, generator=g), torch.randn(Hn, generator=g)
    b[0], b[-1] = 200.0, -200.0                                   # sigmoid 1, and 0 to the power 1 / tau
    buf, decay = Gt.decay_prepare(x.to(DEV), q0, k0, v0, low0, w2.to(DEV), b.to(DEV), Hn, Hv, 0.25, 5.0)
    want = torch.cat([x[:, :Hn] * 0.25, x[:, k0: k0 + Hn], x[:, v0: v0 + Hv]], dim=1)
    z = x[:, low0:].double() @ w2.double() + b.double()
    alpha = torch.exp(-torch.nn.functional.softplus(-z, threshold=1e9) / 5.0)
    assert torch.allclose(buf.cpu(), want, atol=1e-6)
    assert torch.allclose(decay.double().cpu(), alpha, rtol=2e-5, atol=1e-7)
    assert bool((decay[:, 0] == 1.0).all()) and bool((decay[:, -1] < 1e-15).all())


def test_silu_of_column_slices():
    g = torch.Generator().manual_seed(1)
    for width, lo, n in ((40, 8, 24), (13, 3, 7)):
        x = torch.randn(5, width, generator=g) * 20.0
        got = Gt.silu_columns(x.to(DEV)[:, lo: lo + n])
        assert torch.allclose(got.double().cpu(), O.silu(x[:, lo: lo + n].double()), atol=1e-5)


# ------------------------------------------------------------------------------------------------ linear recurrent unit
def _unit(N, blocks, taps, seed, lam_mean=-4.0):
    g = torch.Generator().manual_seed(seed)
    S = N // blocks

    def r(*shape, std=1.0):
        return torch.randn(*shape, generator=g) * std
    return {"conv": r(N, taps, std=0.6), "conv.b": r(N, std=0.5), "x.b": r(N, std=0.5), "y.b": r(N, std=0.5),
            "ra": r(blocks, S, S, std=S ** -0.5), "ri": r(blocks, S, S, std=S ** -0.5), "ra.b": r(blocks, S), "ri.b": r(blocks, S),
            "lam": r(N, std=1.5) + lam_mean}


def _unit_oracle(U, x, y):
    P_ = {k: v.double() for k, v in U.items()}
    u = O.causal_filter(x.double() + P_["x.b"], P_["conv"]) + P_["conv.b"]
    log_a, i = O.lru_gates(u, P_)
    return O.lru_scan(log_a, i * u) * O.gelu_tanh(y.double() + P_["y.b"])


def _unit_step(U, x, y, state, conv_state, info, t2s, single, out=None, scale=1.0):
    N = x.shape[1]
    u = M.conv_silu(x, U["conv"].to(DEV), U["conv.b"].to(DEV), conv_state, info, t2s, U["x.b"].to(DEV), act=False)
    w = torch.stack([U["ra"].transpose(1, 2), U["ri"].transpose(1, 2)]).contiguous().to(DEV)
    b = torch.stack([U["ra.b"].reshape(N), U["ri.b"].reshape(N)]).contiguous().to(DEV)
    a, g = Gt.lru_gates(u, w, b, (-8.0 * torch.nn.functional.softplus(U["lam"])).to(DEV))
    return Gt.lru_scan(a, g, y, U["y.b"].to(DEV), x, state, conv_state, info, single, out, scale)


@pytest.mark.parametrize("N,blocks,taps", [(20, 5, 3), (24, 1, 4), (7, 7, 2), (80, 4, 1), (30, 3, 9), (128, 2, 4), (70, 1, 3)])
def test_recurrent_unit(N, blocks, taps):
    T = 23
    g = torch.Generator().manual_seed(N)
    U, x, y = _unit(N, blocks, taps, N + taps), torch.randn(T, N, generator=g), torch.randn(T, N, generator=g)
    want = _unit_oracle(U, x, y)
    for name, cut in CUTS.items():
        state = torch.full((3, N), 5.0, device=DEV)
        conv = torch.full((3, taps - 1, N), 5.0, device=DEV) if taps > 1 else None
        got = _walk(lambda lo, n, info: _unit_step(U, x[lo: lo + n].to(DEV), y[lo: lo + n].to(DEV), state, conv, info,
                                                   torch.zeros(n, dtype=torch.int32, device=DEV), n == 1), T, cut(T))
        assert torch.allclose(got, want, atol=2e-5, rtol=1e-4), (name, float((got - want).abs().max()))
        assert torch.all(state[[0, 2]] == 5.0)


def test_recurrent_unit_over_a_batch_of_unequal_sequences_into_scaled_slices():
    N, taps = 24, 4
    U = _unit(N, 3, taps, 5)
    g = torch.Generator().manual_seed(6)
    lens, slots = [1, 37, 2, 8], [2, 0, 3, 1]
    xs, ys = [torch.randn(L + 4, N, generator=g) for L in lens], [torch.randn(L + 4, N, generator=g) for L in lens]
    want = [_unit_oracle(U, x, y) for x, y in zip(xs, ys)]
    state, conv = torch.full((5, N), 5.0, device=DEV), torch.full((5, taps - 1, N), 5.0, device=DEV)

    def step(lo, hi):
        rows = [h - l for l, h in zip(lo, hi)]
        first = [sum(rows[:i]) for i in range(4)]
        info = torch.tensor([[f, r, l, s] for f, r, l, s in zip(first, rows, lo, slots)], dtype=torch.int32, device=DEV)
        t2s = torch.arange(4).repeat_interleave(torch.tensor(rows)).to(torch.int32).to(DEV)
        x, y = (torch.cat([t[l:h] for t, l, h in zip(ts, lo, hi)]).to(DEV) for ts in (xs, ys))
        wide = torch.full((sum(rows), N + 8), 7.0, device=DEV)
        _unit_step(U, x, y, state, conv, info, t2s, max(rows) == 1, wide[:, 8:], 0.3)
        assert torch.all(wide[:, :8] == 7.0)
        return [wide[f: f + r, 8:].double().cpu() for f, r in zip(first, rows)]
    got = [[t] for t in step([0] * 4, lens)]
    for i in range(4):
        for lst, t in zip(got, step([L + i for L in lens], [L + i + 1 for L in lens])):
            lst.append(t)
    for lst, w in zip(got, want):
        assert torch.allclose(torch.cat(lst), 0.3 * w, atol=2e-5, rtol=1e-4)
    assert torch.all(state[4] == 5.0) and torch.all(conv[4] == 5.0)


def test_input_bias_starts_with_the_sequence():
    """Filter taps of one and inputs of zero: the first token sees the input bias once, the second twice, from the third on
    three times -- positions before the start carry no bias."""
    x, w, b = torch.zeros(5, 2), torch.ones(2, 3), torch.tensor([1.0, -2.0])
    for cuts in ([5], [1] * 5, [2, 3]):
        state = torch.full((2, 2, 2), 4.0, device=DEV)

        def run(lo, n, info):
            r = x[lo: lo + n].to(DEV)
            u = M.conv_silu(r, w.to(DEV), None, state, info, torch.zeros(n, dtype=torch.int32, device=DEV), b.to(DEV), act=False)
            M.conv_state_update(r, state, info)
            return u
        got = _walk(run, 5, cuts)
        assert torch.equal(got, torch.tensor([1.0, 2.0, 3.0, 3.0, 3.0], dtype=F64)[:, None] * b.double())


def test_slow_channels_keep_their_state_and_small_writes_keep_their_scale():
    """lam = -16 gives 1 - a of about 1e-6: sqrt(1 - a^2) must not lose its digits, and the first token's write is there 400 tokens
    later; lam = +3 forgets it at once."""
    T, N = 400, 2
    U = {"conv": torch.tensor([[1.0]] * N), "conv.b": torch.zeros(N), "x.b": torch.zeros(N), "y.b": torch.full((N,), 3.0),
         "ra": torch.zeros(1, N, N), "ri": torch.zeros(1, N, N), "ra.b": torch.zeros(1, N), "ri.b": torch.full((1, N), 30.0),
         "lam": torch.tensor([-16.0, 3.0])}
    x, y = torch.zeros(T, N), torch.zeros(T, N)
    x[0] = 1.0
    want = _unit_oracle(U, x, y)
    assert want[T - 1, 0] > 1e-4 and want[T - 1, 1] < 1e-30
    for cuts in ([T], [150, 2] + [1] * 248):
        state = torch.full((3, N), 5.0, device=DEV)
        got = _walk(lambda lo, n, info: _unit_step(U, x[lo: lo + n].to(DEV), y[lo: lo + n].to(DEV), state, None, info,
                                                   torch.zeros(n, dtype=torch.int32, device=DEV), n == 1), T, cuts)
        assert torch.allclose(got[:, 0], want[:, 0], rtol=1e-4) and got[T - 1, 1] < 1e-30


# ------------------------------------------------------------------------------------------------ feed-forwards
@pytest.mark.parametrize("E,K,groups,keep", [(12, 3, 4, 2), (8, 2, 2, 1), (16, 4, 8, 3), (6, 2, 6, 2), (5, 3, 1, 1), (8, 8, 4, 4), (64, 6, 8, 4),
                                             (3, 1, 3, 1)])
def test_experts_of_the_groups_with_the_two_best_sums(E, K, groups, keep):
    g = torch.Generator().manual_seed(E)
    z, corr = torch.randn(41, E, generator=g) * 2, torch.randn(E, generator=g) - 1.5     # most choice scores are negative
    sc, assign, offs, counts = moe_ops.top_k_gating(z.to(DEV), K, renormalize=False, score_function="sigmoid", correction=corr.to(DEV),
                                                    n_groups=groups, keep_groups=keep, group_rank="top2")
    s = torch.sigmoid(z.double())
    for t in range(z.shape[0]):
        want = O.choose_experts(s[t], corr.double(), groups, keep, K)
        assert assign[t].tolist() == want
        assert torch.allclose(sc[t].double().cpu(), s[t, want], atol=1e-6)
    assert counts.sum() == 41 * K


def test_rank_by_two_best_differs_from_rank_by_best_and_from_softmax():
    """Group 0 has the best expert, group 1 the better pair; the weights stay the sigmoids themselves."""
    z = torch.tensor([[3.0, -9.0, 2.0, 1.9]])
    kw = dict(correction=torch.zeros(4, device=DEV), n_groups=2, keep_groups=1)
    _, a, _, _ = moe_ops.top_k_gating(z.to(DEV), 2, renormalize=False, score_function="sigmoid", group_rank="top2", **kw)
    assert a.tolist() == [[2, 3]]
    s, a, _, _ = moe_ops.top_k_gating(z.to(DEV), 2, renormalize=False, score_function="sigmoid", group_rank="max", **kw)
    assert a.tolist() == [[0, 1]] and torch.allclose(s.cpu(), torch.sigmoid(z[:, :2]), atol=1e-6)
    s, a, _, _ = moe_ops.top_k_gating(z.to(DEV), 2, scale=2.0, **kw)              # the softmax form divides by the winners' sum
    p = torch.softmax(z, -1)[:, :2]
    assert a.tolist() == [[0, 1]] and torch.allclose(s.cpu(), 2.0 * p / p.sum(), atol=1e-6)


def test_expert_layer_alone():
    g = torch.Generator().manual_seed(3)
    W, E, Fe, K = 24, 12, 10, 3
    moe = heuristics.instantiate_moe(DSMoEConfig(
        max_tokens=64, model_dim=W, intermediate_features=Fe, n_experts=E, top_k=K, input_dtype=DtypeEnum.fp32,
        output_dtype=DtypeEnum.fp32, activation=ActivationType.SiGLU, score_function="sigmoid", router_dtype=DtypeEnum.fp32,
        score_correction=True, n_groups=4, keep_groups=2, group_rank="top2", plain_group_scores=True), None)
    P_ = {"router": torch.randn(E, W, generator=g), "correction": torch.randn(E, generator=g)}
    for e in range(E):
        P_[f"e{e}.gate"], P_[f"e{e}.up"] = (torch.randn(Fe, W, generator=g) / W ** 0.5 for _ in range(2))
        P_[f"e{e}.down"] = torch.randn(W, Fe, generator=g) / Fe ** 0.5
    h = torch.randn(17, W, generator=g)
    want = O.expert_ff(h.double(), {k: v.double() for k, v in P_.items()},
                       {"router": {"experts": E, "top": K, "groups": {"count": 4, "keep": 2}}})
    w1 = torch.stack([torch.cat([P_[f"e{e}.gate"], P_[f"e{e}.up"]]) for e in range(E)]).to(DEV)
    w2 = torch.stack([P_[f"e{e}.down"] for e in range(E)]).to(DEV)
    for n in (17, 1):
        got = moe(h[:n].to(DEV), P_["router"].to(DEV), w1, w2, correction=P_["correction"].to(DEV))
        assert torch.allclose(got.double().cpu(), want[:n], atol=1e-5)


@pytest.mark.parametrize("ff", [16, 11])
def test_clamped_activation_at_and_beyond_its_limits(ff):
    """gate: clamped from above only; up: on both sides, then plus one."""
    x = torch.linspace(-4.0, 4.0, 6 * 2 * ff).view(6, 2 * ff)[:, torch.randperm(2 * ff, generator=torch.Generator().manual_seed(ff))]
    got = M.gated_act_rows(x.to(DEV), "clamped_swish", 1.25).double().cpu()
    gte, up = x[:, :ff].double().clamp(max=1.25), x[:, ff:].double().clamp(min=-1.25, max=1.25)
    assert torch.allclose(got, gte * torch.sigmoid(1.702 * gte) * (up + 1.0), atol=1e-5)


# ------------------------------------------------------------------------------------------------ layers and the stack
@pytest.mark.parametrize("layer", [LIGHT, UNIT, WIN], ids=["lightning", "parallel", "parallel_2"])
@pytest.mark.parametrize("mlp", [None, DENSE, MOE], ids=["alone", "dense", "experts"])
def test_one_layer_of_each_kind(layer, mlp):
    cfg = make_cfg([dict(layer, mlp=mlp)])
    W = O.random_weights(cfg, seed=1)
    toks = tokens(23, cfg["vocab"], 2)
    want = O.forward(cfg, W, toks)
    eng = make_engine(cfg, W)
    close(feed(eng, 1, toks, [len(toks)]), want)
    close(feed(eng, 2, toks, [3, 1, 2]), want)


@pytest.mark.parametrize("layer", [UNIT, WIN], ids=["parallel", "parallel_2"])
@pytest.mark.parametrize("scales", [(1.0, 0.0), (0.0, 1.0), (-0.5, 2.0)])
def test_each_half_of_a_pair_with_its_factor(layer, scales):
    layer = copy.deepcopy(dict(layer, mlp=None))
    layer["mixer"]["left_scale"], layer["mixer"]["right_scale"] = scales
    cfg = make_cfg([layer])
    W = O.random_weights(cfg, seed=2)
    toks = tokens(19, cfg["vocab"], 3)
    eng = make_engine(cfg, W)
    close(feed(eng, 1, toks, [5, 1, 13]), O.forward(cfg, W, toks))


def test_stream_after_every_layer(stack):
    W, toks, _ = stack
    handed = []
    O.forward(STACK, W, toks, handed)
    eng = make_engine(STACK, W)
    eng.model().layer_outputs = []
    feed(eng, 1, toks, [len(toks)])
    assert len(handed) == len(eng.model().layer_outputs) == 5
    for got, want in zip(eng.model().layer_outputs, handed):
        assert torch.allclose(got.double().cpu(), want, atol=2e-4, rtol=1e-4)


def test_embedding_factor_and_soft_cap():
    for scale, cap in ((1.0, 50.0), (7.0, 0.5)):
        cfg = make_cfg([LIGHT], scale=scale, cap=cap)
        W = O.random_weights(cfg, seed=3)
        toks = tokens(9, cfg["vocab"], 4)
        got = feed(make_engine(cfg, W), 1, toks, [9])
        close(got, O.forward(cfg, W, toks))
        assert got.abs().max() <= cap


@pytest.mark.parametrize("size", [1, 2, 7, 12])
def test_what_lies_just_outside_the_window_does_not_matter_and_just_inside_does(size):
    """One pair whose recurrent half is muted and whose filters pass the current token only: the last position's logits change with
    the token ``size - 1`` back and not with the token ``size`` back, in a prompt and decoded alone."""
    layer = copy.deepcopy(dict(WIN, mlp=None))
    layer["mixer"]["left"].update(mask={"size": size}, scale=2.0)
    layer["mixer"]["right_scale"] = 0.0
    cfg = make_cfg([layer])
    W = O.random_weights(cfg, seed=13)
    for n in "qkv":
        w = torch.zeros_like(W[f"l0.mix.left.{n}.conv"])
        w[:, -1] = 1.0
        W[f"l0.mix.left.{n}.conv"] = w
    toks = tokens(21, cfg["vocab"], 14)
    base = O.forward(cfg, W, toks)
    eng, uid = make_engine(cfg, W, max_live=2), 0
    for back, matters in ((size, False), (size - 1, True), (size + 3, False)):
        other = list(toks)
        other[-1 - back] = (other[-1 - back] + 17) % cfg["vocab"]
        want = O.forward(cfg, W, other)
        assert bool((want[-1] - base[-1]).abs().max() > 1e-3) == matters
        for sizes in ([len(toks)], [len(toks) - 3, 1], [4, 2, 5]):
            uid += 1
            got = feed(eng, uid, other, sizes)
            close(got, want)
            assert bool((got[-1] - base[-1]).abs().max() > 1e-3) == matters
            eng.flush(uid)


def test_far_keys_and_old_writes_decide_the_logits():
    """Attention with its score scale raised, so that single keys carry most of a query's weight wherever they lie among hundreds,
    and recurrences that barely decay: prompt rows, portions cut at page and window borders and beside them, and decode tokens
    follow the plain evaluation."""
    unit, win, light = (copy.deepcopy(dict(x, mlp=None)) for x in (UNIT, WIN, LIGHT))
    unit["mixer"]["left"]["scale"] = 4.0
    win["mixer"]["left"].update(scale=3.0, mask={"size": 64})
    win["mixer"]["right"]["tau"] = 400.0
    light["mixer"]["decay"] = [0.999, 0.9999, 0.99]
    cfg = make_cfg([unit, win, light], vocab=31)
    W = O.random_weights(cfg, seed=21)
    W["l0.mix.right.lam"] = torch.full_like(W["l0.mix.right.lam"], -9.0)
    toks = tokens(300, cfg["vocab"], 22)
    want = O.forward(cfg, W, toks)
    eng = make_engine(cfg, W, block_size=8, blocks=128, max_tokens=320)
    close(feed(eng, 1, toks, [len(toks)]), want)
    close(feed(eng, 2, toks, [245] + [1] * 55), want)
    close(feed(eng, 3, toks, [64, 37, 3, 2, 40, 4, 127, 1, 7, 15]), want)
    other = tokens(40, cfg["vocab"], 23) + toks[40:]                 # another beginning gives other logits at the end
    assert (O.forward(cfg, W, other)[-1] - want[-1]).abs().max() > 1e-2


# ------------------------------------------------------------------------------------------------ cache, state, batches
def test_prefill_equals_token_by_token_decoding(stack):
    W, toks, want = stack
    eng = make_engine(STACK, W)
    close(feed(eng, 1, toks, [len(toks)]), want)
    close(feed(eng, 2, toks, [1]), want)


@pytest.mark.parametrize("sizes", [[2], [3, 5], [7, 1, 1, 2], [16, 2, 9], [40, 1], [1, 2]])
def test_prompt_portions(stack, sizes):
    W, toks, want = stack
    eng = make_engine(STACK, W)
    close(feed(eng, 1, toks, sizes), want)


def test_unequal_requests_in_one_batch_equal_each_alone():
    W = O.random_weights(STACK, seed=9)
    reqs = {u: tokens(n, STACK["vocab"], 10 + u) for u, n in ((1, 19), (2, 3), (3, 31), (4, 8))}
    want = {u: O.forward(STACK, W, t) for u, t in reqs.items()}
    eng = make_engine(STACK, W)
    at = {u: 0 for u in reqs}
    got = {u: [] for u in reqs}
    plan = [{1: 5, 3: 2}, {1: 1, 2: 3, 3: 9, 4: 2}, {1: 13, 3: 1, 4: 1}, {3: 1, 4: 1}, {3: 1, 4: 4}, {3: 17}]
    for step in plan:                                              # 2 is left out, 1 ends, a step of single tokens only
        uids = list(step)
        toks = [torch.tensor(reqs[u][at[u]: at[u] + n]) for u, n in step.items()]
        out = eng.put(uids, toks, logit_positions=[list(range(n)) for n in step.values()]).double().cpu()
        k = 0
        for u, n in step.items():
            got[u].append(out[k: k + n])
            k, at[u] = k + n, at[u] + n
    for u in reqs:
        assert at[u] == len(reqs[u])
        close(torch.cat(got[u]), want[u])


def test_a_step_that_asks_for_no_logits_still_advances(stack):
    W, toks, want = stack
    eng = make_engine(STACK, W)
    for lo, n in ((0, 9), (9, 1), (10, 2)):
        out = eng.put([1], [torch.tensor(toks[lo: lo + n])], logit_positions=[[]])
        assert out.shape == (0, STACK["vocab"])
    rest = eng.put([1], [torch.tensor(toks[12:])], logit_positions=[list(range(len(toks) - 12))]).double().cpu()
    close(rest, want[12:])


def test_pages_and_state_slots_are_reused():
    """As many pages as the longest request and its neighbour need, two state slots: every later request gets pages and a
    slot that an earlier one filled, in another order, and must come out as if alone -- also one shorter than the filters."""
    W = O.random_weights(STACK, seed=3)
    eng = make_engine(STACK, W, blocks=10, block_size=4, max_live=2)
    for i, n in enumerate((20, 23, 1, 26, 2, 29)):
        toks = tokens(n, STACK["vocab"], 20 + i)
        other = tokens(6, STACK["vocab"], 40 + i)
        eng.put([100 + i], [torch.tensor(other)])                 # a neighbour that holds the other slot and two pages
        got = feed(eng, i, toks, [7, 1, 2] if i % 2 else [1, 1, 4])
        close(got, O.forward(STACK, W, toks))
        eng.flush(i)
        eng.flush(100 + i)
        assert eng.free_blocks == 10


def test_long_decoding(stack):
    W, _, _ = stack
    toks = tokens(150, STACK["vocab"], 6)
    want = O.forward(STACK, W, toks)
    eng = make_engine(STACK, W)
    close(feed(eng, 1, toks, [9] + [1] * 200), want)


ODD = [
    # nothing a multiple of 8, single heads, a window of one token, one tap, one block, one group, one expert of three, tau 1
    (make_cfg([{"type": "parallel_2",
                "mixer": {"left": {"dim": 5, "heads": 1, "kv_heads": 1, "vdim": 3, "conv": 1, "mask": {"size": 1}, "scale": 1.7,
                                   "rot": {"base": 77.0, "dims": 4}},
                          "right": {"dim": 7, "heads": 1, "vdim": 3, "tau": 1.0}, "left_scale": 1.0, "right_scale": 1.0},
                "mlp": {"kind": "moe", "expert": {"ff": 9}, "router": {"experts": 3, "groups": {"count": 1, "keep": 1}, "top": 1}}},
               {"type": "parallel",
                "mixer": {"left": {"dim": 6, "heads": 3, "kv_heads": 1, "vdim": 5, "scale": 0.9, "rot": {"base": 12.0, "dims": 2}},
                          "right": {"width": 11, "blocks": 1, "conv": 1}, "left_scale": 0.3, "right_scale": 1.0},
                "mlp": {"ff": 11, "kind": "dense", "limit": 2.0}}], width=10, vocab=17, eps=1e-3), 1),
    # values wider than keys, key sizes above 32, long filters, groups of one expert, more heads than the width has words
    (make_cfg([{"type": "lightning", "mixer": {"dim": 36, "heads": 1, "vdim": 50, "decay": [0.97]}, "mlp": None},
               {"type": "parallel_2",
                "mixer": {"left": {"dim": 16, "heads": 8, "kv_heads": 8, "vdim": 40, "conv": 7, "mask": {"size": 16}, "scale": 0.2,
                                   "rot": {"base": 1e4, "dims": 8, "scaling": {"factor": 16.0, "original": 32, "fast": 4.0, "slow": 1.0}}},
                          "right": {"dim": 20, "heads": 2, "vdim": 4, "tau": 30.0}, "left_scale": 0.5, "right_scale": 0.8},
                "mlp": {"kind": "moe", "expert": {"ff": 16}, "router": {"experts": 4, "groups": {"count": 4, "keep": 3}, "top": 2}}},
               {"type": "parallel",
                "mixer": {"left": {"dim": 12, "heads": 2, "kv_heads": 2, "vdim": 20, "scale": 0.4, "rot": {"base": 50.0, "dims": 12}},
                          "right": {"width": 64, "blocks": 64, "conv": 5}, "left_scale": 0.8, "right_scale": 0.5}, "mlp": None}],
              width=64, vocab=29), 8),
    # a stack of one kind each; windows longer than the sequence
    (make_cfg([{"type": "parallel_2",
                "mixer": {"left": {"dim": 4, "heads": 2, "kv_heads": 1, "vdim": 4, "conv": 2, "mask": {"size": 500}, "scale": 0.5,
                                   "rot": {"base": 30.0, "dims": 4}},
                          "right": {"dim": 4, "heads": 4, "vdim": 4, "tau": 8.0}, "left_scale": 0.5, "right_scale": 0.5},
                "mlp": None}] * 2, width=8, vocab=11), 3),
    (make_cfg([dict(LIGHT, mlp=MOE), dict(LIGHT, mlp=None)], width=16, vocab=23, scale=1.0, cap=1.0), 4),
]


@pytest.mark.parametrize("cfg,rank", ODD, ids=["ones_everywhere", "wide_values_long_filters", "pairs_only", "lightning_only"])
def test_other_sizes(cfg, rank):
    W = O.random_weights(cfg, seed=8, rank=rank)
    toks = tokens(21, cfg["vocab"], 9)
    want = O.forward(cfg, W, toks)
    eng = make_engine(cfg, W, block_size=8)
    close(feed(eng, 1, toks, [len(toks)]), want)
    close(feed(eng, 2, toks, [4, 1, 2]), want)


def test_configuration_is_read_into_the_layer_specs():
    from shuffle_exchange_b200.inference.v2.checkpoint.huggingface_engine import PlainModelConfig
    from shuffle_exchange_b200.inference.v2.model_implementations.sudupel import SudupelPolicy
    spec = SudupelPolicy(PlainModelConfig(STACK)).spec(PlainModelConfig(STACK))
    light, win, unit, win2, _ = spec.layers
    assert (light.kind, light.n_heads, light.key_dim, light.value_dim, light.head_decay) == ("lightning", 3, 8, 12, (0.55, 0.9, 0.995))
    assert (light.ff_kind, light.ff_activation, light.ff_limit, light.ff_dim, unit.ff_dim) == ("gated", "clamped_swish", 0.8, 24, 0)
    a, b = unit.parts
    assert (a.kind, a.n_heads, a.n_heads_kv, a.key_dim, a.value_dim, a.attn_scale, a.rot_dims, a.rot_base, a.rot_scaling, a.window) == (
        "rotary_attention", 4, 2, 8, 6, 0.4, 6, 300.0, (3.0, 64.0, 8.0, 1.0), 0)
    assert a.qk_row_norm and a.unit_sink and not a.rot_interleaved
    assert (b.kind, b.n_heads, b.key_dim, b.conv_taps, b.decay_rate, unit.pair_scales) == ("lru", 5, 4, 3, 8.0, (0.7, 0.9))
    a, b = win.parts
    assert (a.kind, a.conv_taps, a.window, a.rot_scaling, a.qk_norm_weight, a.unit_sink, a.qk_row_norm) == (
        "attention", 4, 7, None, True, False, False)
    assert (b.kind, b.n_heads, b.key_dim, b.value_dim, b.decay_tau, win.pair_scales) == ("channel_decay", 3, 4, 8, 5.0, (1.3, 0.4))
    assert (win.ff_kind, win.n_experts, win.top_k, win.moe_groups, win.moe_keep_groups, win.moe_group_rank, win.moe_score) == (
        "moe", 12, 3, 4, 2, "top2", "sigmoid")
    assert win.moe_plain_scores and win.moe_correction and win2.ff_kind == "gated"
    assert (spec.block_form, spec.norm_weight_offset, spec.embed_scale, spec.logit_softcap, spec.norm_eps) == (
        "sandwich", 1.0, 3.0, 6.0, 1e-5)
    bad = copy.deepcopy(STACK)
    bad["layers"][1]["mixer"]["left"]["conv"] = 3
    with pytest.raises(ValueError, match="conv"):
        make_engine(bad, O.random_weights(STACK))
    bad = copy.deepcopy(STACK)
    bad["layers"][2]["mixer"]["right"]["blocks"] = 3
    with pytest.raises(ValueError, match="equal blocks"):
        make_engine(bad, O.random_weights(STACK))


def test_every_checkpoint_tensor_is_used(monkeypatch):
    from shuffle_exchange_b200.inference.v2.model_implementations.inference_policy_base import ContainerMap
    left = []
    monkeypatch.setattr(ContainerMap, "set_unmapped_params", lambda self, names: left.append(list(names)))
    make_engine(STACK, O.random_weights(STACK, seed=2))
    assert left == [[]]


def test_bf16_serving_stays_near_the_exact_evaluation(stack):
    W, toks, want = stack
    eng = make_engine(STACK, W, dtype=torch.bfloat16)
    for uid, sizes in ((1, [len(toks)]), (2, [5, 1, 2])):
        err = row_errors(feed(eng, uid, toks, sizes), want)        # a close choice of experts may fall the other way in a few rows
        assert err.median() < 0.04 and err.max() < 0.5


# ------------------------------------------------------------------------------------------------ generation
def _check_greedy(prompt, out, W, cfg):
    seq = list(prompt)
    for tok in out:
        logits = O.forward(cfg, W, seq)[-1]
        top2 = logits.topk(2).values
        if top2[0] - top2[1] > 1e-3:                           # a near tie may go either way in 32-bit
            assert tok == int(logits.argmax())
        seq.append(tok)


def test_greedy_generation_through_the_scheduler():
    W = O.random_weights(STACK, seed=12)
    prompts = [tokens(n, STACK["vocab"], 30 + n) for n in (5, 17, 2, 9, 12)]          # five requests, four may be live
    eng = make_engine(STACK, W, blocks=40, block_size=4, max_live=4, max_tokens=16)
    got = generate(eng, prompts, max_new_tokens=6, max_batch_tokens=16, max_prompt_portion=7)
    for p, out in zip(prompts, got):
        _check_greedy(p, out, W, STACK)
        assert len(out) == 6
    assert eng.free_blocks == 40 and eng._state_manager.n_tracked_sequences == 0


def write_checkpoint(folder, cfg, W):
    """``config.json`` + ``model.safetensors`` (bf16): 8-byte header length, JSON header, tensor bytes."""
    with open(folder / "config.json", "w") as f:
        json.dump(cfg, f)
    meta, blobs, off = {}, [], 0
    for name, t in W.items():
        b = t.to(torch.bfloat16).contiguous().view(torch.int16).numpy().tobytes()
        meta[name] = {"dtype": "BF16", "shape": list(t.shape), "data_offsets": [off, off + len(b)]}
        blobs.append(b)
        off += len(b)
    header = json.dumps(meta).encode()
    with open(folder / "model.safetensors", "wb") as f:
        f.write(struct.pack("<Q", len(header)) + header + b"".join(blobs))


def _run_command(cmd, stdin=None):
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    r = subprocess.run([sys.executable, os.path.join(root, "bin", cmd[0]), *cmd[1:]], input=stdin, capture_output=True,
                       text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    return r.stdout.splitlines()


def test_command_line_generation_from_a_checkpoint_folder(tmp_path):
    W = O.random_weights(STACK, seed=14)
    write_checkpoint(tmp_path, STACK, W)
    prompts = [[5, 17, 3], [9, 9, 1, 2, 3, 4, 5, 6, 7]]
    cmd = ["sxb_generate", "--model", str(tmp_path), "--max-new-tokens", "4", "--dtype", "float32"]
    for p in prompts:
        cmd += ["--prompt", ",".join(map(str, p))]
    lines = [json.loads(x) for x in _run_command(cmd) if x.startswith("{")]
    assert [x["prompt"] for x in lines] == prompts
    for p, x in zip(prompts, lines):
        _check_greedy(p, x["generated"], W, STACK)
        assert len(x["generated"]) == 4


def test_replaying_a_schedule_of_steps_from_a_checkpoint_folder(tmp_path):
    """``bin/trace_run``: five requests through a pool of four 64-token pages and four state slots -- portions beside single
    tokens, a request left out of a step, requests that end and whose pages and slot the next one takes; every wanted position
    must equal the plain evaluation of its request alone."""
    import numpy as np
    W = O.random_weights(STACK, seed=15)
    model = tmp_path / "model"
    model.mkdir()
    write_checkpoint(model, STACK, W)
    reqs = {name: tokens(n, STACK["vocab"], 50 + n) for name, n in (("a", 40), ("b", 9), ("c", 23), ("d", 1), ("e", 30))}
    plan = [({"a": 17, "b": 2}, []), ({"a": 3, "b": 7, "c": 5, "d": 1}, ["b", "d"]), ({"a": 1, "c": 2, "e": 11}, []),
            ({"a": 19, "e": 1}, ["a"]), ({"c": 1, "e": 1}, []), ({"c": 15, "e": 17}, ["c", "e"])]
    at = {k: 0 for k in reqs}
    steps, wanted = [], []
    for i, (portion, end) in enumerate(plan):
        entries = []
        for name, n in portion.items():
            want = sorted({0, n - 1, n // 2})
            entries.append({"id": name, "tokens": reqs[name][at[name]: at[name] + n], "want": want})
            wanted += [(i, name, at[name] + w) for w in want]
            at[name] += n
        steps.append(json.dumps({"step": i, "entries": entries, "end": end}))
    assert at == {k: len(v) for k, v in reqs.items()}
    out = tmp_path / "out"
    cmd = ["trace_run", "--model", str(model), "--dtype", "float32", "--out", str(out), "--max-tokens", "256"]
    lines = _run_command(cmd + ([] if torch.cuda.is_available() else ["--device", "cpu"]), "\n".join(steps) + "\n")
    assert [x for x in lines if x.startswith("done")] == [f"done {i}" for i in range(len(plan))]
    full = {name: O.forward(STACK, W, t) for name, t in reqs.items()}
    got = {i: torch.from_numpy(np.fromfile(out / f"{i}.f32", dtype="<f4").reshape(-1, STACK["vocab"])).double()
           for i in range(len(plan))}
    row = {i: 0 for i in got}
    for i, name, p in wanted:
        close(got[i][row[i]: row[i] + 1], full[name][p: p + 1])
        row[i] += 1
    assert all(row[i] == got[i].shape[0] for i in got)
